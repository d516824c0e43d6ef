"""Vikupel through the engine (scheduler bookkeeping, page / state-slot managers, batch builder, runner) against the plain
oracle in vikupel_oracle.py: mechanisms alone, chunking, batching, re-use of pages and slots, far keys, page borders and
window edges, the loop, the per-layer token input, degenerate sizes, greedy generation. Runs on the CPU path in fp32;
test_vikupel_gpu.py repeats the scenarios on the kernels."""

import numpy as np
import pytest
import torch

import vikupel_oracle as oracle
import vikupel_util as U

TOL = 2e-4
EPS = 1e-5


def toks(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


CONFIGS = {
    # every mixer, in and outside a loop; a layer without feed-forward
    "mixed": U.make_config([U.turned(mlp=U.dense()), U.mamba(mlp=U.dense(20)), U.window(mlp=U.dense(16)),
                            U.mamba(heads=6, groups=3, state=5, vdim=4, conv=3, norm_groups=4, mlp=None),
                            U.turned(heads=3, kv_heads=3, dim=6, vdim=10, rot_dims=6, mlp=U.dense(9))],
                           loop=(1, 4, 2)),
    # no loop, no token side; partial rotation without scaling; a window of two
    "plain": U.make_config([U.window(heads=6, kv_heads=3, dim=4, vdim=10, size=2, mlp=None),
                            U.turned(heads=6, kv_heads=2, dim=10, vdim=4, rot_dims=4, scaling=None, mlp=U.dense(8)),
                            U.mamba(heads=2, groups=1, state=12, vdim=10, conv=2, norm_groups=1, mlp=U.dense(8))],
                           side=0, mult=1.0),
    # no recurrent layer at all, the whole stack in the loop
    "pages_only": U.make_config([U.window(size=9, mlp=U.dense()), U.turned(mlp=U.dense())], loop=(0, 2, 3), mult=0.3),
    # no paged layer at all
    "state_only": U.make_config([U.mamba(mlp=U.dense()), U.mamba(conv=2, mlp=None)], loop=(1, 2, 4)),
    # sizes of one, values that other models make equal or 1
    "ones": U.make_config([U.mamba(heads=1, groups=1, state=1, vdim=1, conv=1, norm_groups=1, mlp=U.dense(1)),
                           U.window(heads=1, kv_heads=1, dim=1, vdim=1, size=1, scale=1.0, mlp=U.dense(3)),
                           U.turned(heads=2, kv_heads=1, dim=2, vdim=2, rot_dims=2, scale=1.0,
                                    scaling={"factor": 1.0, "high": 1.0, "low": 1.0, "original": 8},
                                    mlp=U.dense(2))],
                          width=8, vocab=17, side=1, mult=1.0, loop=(0, 1, 1)),
}


@pytest.fixture(scope="module")
def models():
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        w = U.random_weights(cfg, seed=30 + i)
        out[name] = (cfg, w, U.save_model(cfg, w))
    return out


# -- each mechanism alone, against its own oracle function -----------------------------------------------------
def mixer_alone(layer_cfg, seed, n=19, cuts=((19,), (7, 1, 1, 2, 8), (2,) * 9 + (1,), (1,) * 19), page_size=4,
                device="cpu", dtype=torch.float32, width=20):
    w = U.random_weights(U.make_config([layer_cfg], width=width), seed)
    m = U.build_mixer(layer_cfg, w, width, device, dtype)
    h = torch.randn(n, width, generator=torch.Generator().manual_seed(seed)).bfloat16().float()
    want = U.oracle_mixer(h, layer_cfg, w).float()
    return want, [U.drive_mixer(m, h, list(c), page_size, device, dtype) for c in cuts]


MIXERS = {
    "mamba_groups": U.mamba(),
    "mamba_one_group_ff": U.mamba(heads=3, groups=1, state=5, vdim=8, conv=3, norm_groups=3, mlp=U.dense(7)),
    "mamba_no_taps": U.mamba(heads=2, groups=2, state=1, vdim=3, conv=1, norm_groups=1),
    "mamba_five_taps": U.mamba(conv=5, norm_groups=12),
    "window": U.window(),
    "window_one_kv_head_ff": U.window(heads=5, kv_heads=1, dim=3, vdim=7, size=1, mlp=U.dense(5)),
    "window_wider_than_all": U.window(heads=2, kv_heads=2, size=500),
    "turned": U.turned(),
    "turned_unscaled_whole": U.turned(heads=6, kv_heads=3, dim=6, vdim=2, rot_dims=6, scaling=None, mlp=U.dense(5)),
    "turned_nothing_rotated_in_the_keys": U.turned(rot_dims=0, scaling=None),
}


@pytest.mark.parametrize("name", sorted(MIXERS))
def test_mixer_alone(name):
    want, outs = mixer_alone(MIXERS[name], 40 + len(name))
    for o in outs:
        assert torch.allclose(o, want, atol=1e-4, rtol=1e-4), (o - want).abs().max()


def test_frequency_bands():
    """Short waves keep their frequency, long ones are divided, those between are blended; all three kinds occur."""
    from gllm_b200.ops import ref
    sc = {"factor": 4.0, "high": 8.0, "low": 2.0, "original": 256}
    f = ref.banded_rotary_frequencies(32, 1000.0, sc)
    base = ref.banded_rotary_frequencies(32, 1000.0)
    want = torch.tensor(oracle.frequencies(32, 1000.0, sc), dtype=torch.float64)
    assert torch.allclose(f, want, rtol=1e-12)
    ratio = base / f
    assert (ratio < 1 + 1e-9).any() and (ratio > 4 - 1e-9).any() and ((ratio > 1.01) & (ratio < 3.99)).any()
    flat = ref.banded_rotary_frequencies(8, 50.0, {"factor": 2.0, "high": 3.0, "low": 3.0, "original": 30})
    assert torch.isfinite(flat).all()


def test_rotation_keeps_relative_scores_and_values():
    """Values rotated by j and turned back by i leave only i - j: shifting all positions changes nothing."""
    layer = U.turned(heads=2, kv_heads=1, rot_dims=8, scaling=None)
    w = U.random_weights(U.make_config([layer]), 5)
    m, t = layer["mixer"], 12
    h = torch.randn(t, 20, generator=torch.Generator().manual_seed(2)).double()
    a = oracle.rotated_value_attention(h, m, w, "l0.mix.", EPS)
    f = oracle.frequencies(m["vdim"], m["rot"]["base"])
    assert max(f) == 1.0 and len(f) == m["vdim"] // 2
    mixer = U.build_mixer(layer, w, 20)
    assert torch.allclose(U.drive_mixer(mixer, h.float(), [t]), a.float(), atol=1e-4)
    # a distance-dependent effect: the same attention without rotated values differs
    plain = oracle.softmax_heads(
        oracle.rms(oracle.rotate(oracle.linear(h, w, "l0.mix.q").reshape(t, 2, 8), oracle.frequencies(8, 90.0)), EPS),
        oracle.rms(oracle.rotate(oracle.linear(h, w, "l0.mix.k").reshape(t, 1, 8), oracle.frequencies(8, 90.0)), EPS),
        oracle.linear(h, w, "l0.mix.v").reshape(t, 1, m["vdim"]), m["scale"], oracle.distances(t) >= 0)
    plain = oracle.linear(plain.reshape(t, -1), w, "l0.mix.o")
    assert (plain - a)[1:].abs().max() > 0.1


def test_stream_update_with_a_multiplier_and_without_a_norm():
    from gllm_b200.layers import functional as Fn
    g = torch.Generator().manual_seed(1)
    x, y, w = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g), torch.rand(12, generator=g)
    a = x.clone()
    out = Fn.resid_norm(a, y, None, None, w, EPS, torch.float32, y_mul=0.3)
    assert torch.allclose(a, x + 0.3 * y) and torch.allclose(out, oracle.rms(a.double(), EPS).float() * w, atol=1e-6)
    b = x.clone()
    Fn.resid_norm(b, y, w, None, None, EPS, torch.float32, y_mul=0.3)
    assert torch.allclose(b, x + 0.3 * oracle.rms(y, EPS) * w, atol=1e-6)


def test_gate_comes_before_the_grouped_norm():
    from gllm_b200.ops import ref
    g = torch.Generator().manual_seed(3)
    o, z, w = (torch.randn(4, 12, generator=g) for _ in range(3))
    for parts in (1, 2, 3, 12):
        got = ref.gate_then_norm(o, z, w[0], 12 // parts, EPS)
        want = oracle.gated_norm(o.double(), z.double(), w[0].double(), parts, EPS).float()
        assert torch.allclose(got, want, atol=1e-5)


def test_recurrence_strong_and_weak_decays():
    """Steps far out on both sides of the softplus: a state that vanishes at once and one that never decays."""
    from gllm_b200.ops import ref
    g = torch.Generator().manual_seed(4)
    t, H, G, N, V = 9, 4, 2, 3, 5
    x, b, c = (torch.randn(t, n, generator=g) for n in (H * V, G * N, G * N))
    dt = torch.tensor([[-30.0, 0.0, 4.0, 40.0]]).repeat(t, 1) + torch.randn(t, H, generator=g)
    a_log, bias, d = torch.tensor([0.0, -8.0, 2.0, 1.0]), torch.randn(H, generator=g), torch.randn(H, generator=g)
    qsl, sl = torch.tensor([0, t]), torch.tensor([t])
    got = ref.ssd_scan(x, b, c, dt, -torch.exp(a_log), bias, d, None, None, sl, qsl, H, G, N, V)
    step = torch.log1p(torch.exp(dt.double() + bias.double()))
    want = oracle.ssd_scan(x.double().reshape(t, H, V), b.double().reshape(t, G, N), c.double().reshape(t, G, N), step,
                           a_log.double(), d.double())
    assert torch.allclose(got, want.reshape(t, -1).float(), rtol=1e-4, atol=1e-4)


def test_token_side_reads_the_layers_own_part():
    from gllm_b200.ops import ref
    g = torch.Generator().manual_seed(6)
    z, table = torch.randn(4, 3, generator=g), torch.randn(11, 9, generator=g)
    ids = torch.tensor([7, 0, 10, 7])
    for layer in range(3):
        got = ref.gelu_gate_embed(z, ids, table, 3 * layer)
        want = oracle.gelu_tanh(z.double()) * table.double()[ids][:, 3 * layer:3 * layer + 3]
        assert torch.allclose(got, want.float(), atol=1e-6)


# -- whole models ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_matches_oracle(models, name):
    cfg, w, path = models[name]
    t = toks(37, cfg["vocab"], 1)
    got = U.run_chunks(U.session(path), "a", t, [len(t)])
    assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL


def test_residual_stream_after_every_layer_run(models):
    cfg, w, path = models["mixed"]
    t = toks(15, cfg["vocab"], 2)
    s = U.session(path)
    s.runner.model.trace = []
    U.run_chunks(s, "a", t, [len(t)])
    want = []
    U.expected_logits(cfg, w, t, want)
    assert len(want) == len(s.runner.model.trace) == 8          # 5 layers, three of them twice
    for a, b in zip(s.runner.model.trace, want):
        assert torch.allclose(a, b.float(), atol=1e-3, rtol=1e-4)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token_equals_prefill(models, name):
    cfg, w, path = models[name]
    t = toks(26, cfg["vocab"], 3)
    got = U.run_chunks(U.session(path), "a", t, [])
    assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL


@pytest.mark.parametrize("cuts", [(2,) * 20, (3, 2, 5, 2, 2, 9, 2), (16, 1, 1, 2, 17), (1, 36, 2)])
def test_portions(models, cuts):
    for name in ("mixed", "plain", "ones"):
        cfg, w, path = models[name]
        t = toks(40, cfg["vocab"], 4)
        got = U.run_chunks(U.session(path), "a", t, list(cuts))
        assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL, name


PLAN = [[("a", 13)], [("a", 1), ("b", 7)], [("a", 2), ("b", 1), ("c", 11)], [("a", 4), ("c", 1)],
        [("d", 2), ("b", 3), ("c", 2)], [("c", 1), ("d", 1)], [("e", 9), ("d", 6), ("c", 1)],
        [("e", 1), ("f", 14), ("d", 1)], [("e", 2), ("f", 1)], [("g", 5), ("f", 2), ("e", 1)], [("g", 1)]]


def test_mixed_batch_equals_alone_and_reuses_pages_and_slots(models):
    """Portions beside decoded tokens, requests left out of steps, pages and slots of finished requests used again."""
    for name in ("mixed", "state_only", "pages_only"):
        cfg, w, path = models[name]
        total = {}
        for step in PLAN:
            for k, n in step:
                total[k] = total.get(k, 0) + n
        reqs = {k: toks(n, cfg["vocab"], 50 + i) for i, (k, n) in enumerate(sorted(total.items()))}
        s = U.session(path, max_tokens=72, page_size=4)
        got = U.run_plan(s, reqs, PLAN)
        for k, t in reqs.items():
            assert U.rel_err(got[k], U.expected_logits(cfg, w, t)) < TOL, (name, k)
        mm = s.scheduler.mm
        assert mm.get_num_free_pages() == mm.usable_pages or mm.id_allocator.get_num_used_ids() <= 1


def test_stale_slot_and_page_contents_do_not_leak(models):
    cfg, w, path = models["mixed"]
    s = U.session(path, max_tokens=64, page_size=4)
    cache = s.runner.kv_cache if hasattr(s.runner, "kv_cache") else s.runner.cache
    for group in (cache.k_cache, cache.v_cache, cache.conv_state, cache.ssm_state):
        for x in group:
            if x is not None:
                x.fill_(37.0)
    t = toks(22, cfg["vocab"], 8)
    assert U.rel_err(U.run_chunks(s, "a", t, [1, 2, 5]), U.expected_logits(cfg, w, t)) < TOL


def test_first_tokens_of_a_sequence(models):
    for name in CONFIGS:
        cfg, w, path = models[name]
        s = U.session(path)
        for n in (1, 2, 3, 4, 5):
            t = toks(n, cfg["vocab"], 60 + n)
            for cuts in ([n], [1] * n, [max(n - 1, 1)]):
                got = U.run_chunks(s, "r%d%s" % (n, len(cuts)), t, cuts)
                assert U.rel_err(got, U.expected_logits(cfg, w, t)) < TOL, (name, n, cuts)


def marked_key_probe(kind, n, back, size, page_size, device="cpu", dtype=torch.float32, heads=2, kv_heads=2, dim=32,
                     vdim=4, cuts=None):
    """One attention mixer in which the last query singles out one key. The query map is the key map after a
    permutation of the input, the key maps are orthogonal, inputs have unit length and the scale is large; the last
    token's input is the permuted input of the token `back` places before it.
    -> (oracle, [outputs for several ways of cutting], the oracle with the marked token's input replaced)."""
    g = torch.Generator().manual_seed(back * 7 + page_size)
    width, rot = dim, 2
    if kind == "window":
        layer = U.window(heads, kv_heads, dim, vdim, size, scale=70.0)
    else:
        layer = U.turned(heads, kv_heads, dim, vdim, rot, base=500.0, scaling=None, scale=70.0 / dim)
    w = U.random_weights(U.make_config([layer], width=width), 99)
    wk = torch.stack([torch.linalg.qr(torch.randn(dim, dim, generator=g))[0] for _ in range(kv_heads)])
    if kind != "window":
        wk[:, :rot] = 0                                        # the rotated entries stay out of the scores
    perm = torch.roll(torch.arange(width), 5)                  # query(h) = key(h') with h'[perm] = h
    w["l0.mix.k"] = wk.reshape(-1, width).bfloat16().float()
    w["l0.mix.q"] = wk.repeat_interleave(heads // kv_heads, 0).reshape(-1, width)[:, perm].bfloat16().float()
    if kind == "window":
        w["l0.mix.r1"], w["l0.mix.r2"] = torch.full((heads,), 1.5), torch.full((heads,), 0.5)
    m = U.build_mixer(layer, w, width, device, dtype)
    h = torch.randn(n, width, generator=g)
    h = h / h.norm(dim=-1, keepdim=True)
    tgt = n - 1 - back
    h[n - 1] = h[tgt][perm]                                    # the last query equals the marked token's key
    h = h.bfloat16().float()
    want = U.oracle_mixer(h, layer, w).float()
    h2 = h.clone()
    if back > 0:
        x = torch.randn(width, generator=g)
        h2[tgt] = x / x.norm()
    other = U.oracle_mixer(h2, layer, w).float()
    outs = []
    for c in cuts or [[n], [n - 1, 1], [n - back - 1, 1] + [back] * (back > 0), [max(n - 40, 1)] + [2] * 19]:
        c = [x for x in c if x > 0]
        rest = n - sum(c)
        outs.append(U.drive_mixer(m, h, c + [1] * rest, page_size, device, dtype, pool=1024))
    return want, outs, other


@pytest.mark.parametrize("page_size", [4, 16])
def test_far_keys_and_page_borders(page_size):
    n = 331
    for back in (0, 1, page_size - 1, page_size, page_size + 1, 63, 64, 65, 200, 329, 330):
        want, outs, other = marked_key_probe("turned", n, back, None, page_size)
        if back > 0:          # the oracle's last row rests on the marked key
            assert (want[-1] - other[-1]).abs().max() > 0.05 * want[-1].abs().max(), back
        for o in outs:
            assert torch.allclose(o, want, atol=1e-4 * want.abs().max().item(), rtol=2e-4), (page_size, back)


@pytest.mark.parametrize("size", [1, 2, 33, 64, 100])
def test_window_edges(size):
    """A key just inside the window decides the last row, one just outside does not touch it."""
    n = 150
    for back in (size - 2, size - 1, size, size + 1):
        if back < 0:
            continue
        want, outs, other = marked_key_probe("window", n, back, size, 16)
        moved = (want[-1] - other[-1]).abs().max() / want[-1].abs().max()
        if back > 0:
            assert (moved > 0.05) if back < size else (moved == 0), (size, back, moved)
        for o in outs:
            assert torch.allclose(o, want, atol=1e-4 * want.abs().max().item(), rtol=2e-4), (size, back)


def test_distance_bias_shows():
    layer = U.window(size=12)
    w = U.random_weights(U.make_config([layer]), 7)
    h = torch.randn(16, 20, generator=torch.Generator().manual_seed(7))
    base = U.oracle_mixer(h, layer, w)
    for name in ("r1", "r2"):
        w2 = dict(w)
        w2["l0.mix." + name] = w["l0.mix." + name] * 3
        want = U.oracle_mixer(h, layer, w2)
        assert (want - base).abs().max() > 0.05
        assert torch.allclose(U.drive_mixer(U.build_mixer(layer, w2, 20), h, [5, 1, 2, 8]), want.float(), atol=1e-4)


def test_long_decoding(models):
    """A long prompt, then hundreds of single tokens: the state and the pages go far past the first ones."""
    cfg, w, path = models["mixed"]
    t = toks(260, cfg["vocab"], 11)
    got = U.run_chunks(U.session(path, max_tokens=512, page_size=16), "a", t, [60, 3, 2])
    e = U.row_errs(got, U.expected_logits(cfg, w, t))
    assert np.median(e) < 1e-5 and e.max() < 1e-3       # a few of so many rows amplify fp32 rounding


def test_loop_passes_keep_their_own_cache(models):
    cfg, w, path = models["mixed"]
    s = U.session(path)
    model = s.runner.model
    assert [i for i, _ in model.runs] == oracle.layer_order(cfg) == [0, 1, 2, 3, 1, 2, 3, 4]
    lay = model.cache_layout()
    assert [e["kind"] for e in lay] == ["kv", "linear", "kv", "linear", "linear", "kv", "linear", "kv"]
    # the same stack without the loop is another model
    flat = {k: v for k, v in cfg.items() if k != "loop"}
    t = toks(12, cfg["vocab"], 12)
    assert U.rel_err(U.expected_logits(flat, w, t), U.expected_logits(cfg, w, t)) > 0.05


def test_greedy_generation_through_the_engine(models):
    from gllm_b200.engine.llm_engine import LLM
    cfg, w, path = models["mixed"]
    llm = LLM(path, dtype="float32", page_size=4, maxp=16, maxd=8, num_cpu_pages=64, model_max_length=96,
              log_stats=False, device="cpu", num_state_slots=2)
    prompts = [toks(21, cfg["vocab"], 31), toks(3, cfg["vocab"], 32), toks(9, cfg["vocab"], 33)]
    lens = [7, 12, 5]
    seqs = llm.generate(tokens=prompts, output_lens=lens, temperature=0.0, top_k=1)
    for p, n, s in zip(prompts, lens, seqs):
        cur = list(p)
        for _ in range(n):
            cur.append(int(oracle.forward(cfg, w, cur)[-1].argmax()))
        assert s.token_ids == cur


def test_side_benchmark_configuration_is_served():
    """The layer-like configuration of `bench.py --design vikupel` (scaled down) is a valid model of this design: it
    builds with random weights and generates through the engine."""
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    from benchmarks.vikupel_bench import vikupel_cfg
    from gllm_b200.engine.llm_engine import LLM
    cfg = vikupel_cfg(128, 1, 97, window=12)
    assert [L["type"] for L in cfg["layers"]] == ["mamba2", "attention", "mamba2", "attention_2"]
    cfg["torch_dtype"] = "float32"
    llm = LLM(cfg, load_format="dummy", page_size=4, maxp=16, maxd=4, num_cpu_pages=32, model_max_length=64,
              log_stats=False, device="cpu", num_state_slots=2)
    seqs = llm.generate(tokens=[toks(9, 97, 1), toks(4, 97, 2)], output_lens=[3, 2], temperature=0.0, top_k=1)
    assert [len(s.token_ids) for s in seqs] == [12, 6]
