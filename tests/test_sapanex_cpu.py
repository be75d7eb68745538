"""Sapanex on CPU: the reader of its configuration, every operator's PyTorch statement against the plain oracle, and the engine - scheduler,
pages, pooled rows, state slots, portions, mixed batches, generation - in 32-bit against the oracle's logits."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import sapanex_oracle as oracle
from nanoengine_b200 import Config, LLM, SamplingParams
from nanoengine_b200.models.config import PRESETS, ModelConfig, _yarn_of
from nanoengine_b200.ops import reference as ref
from sapanex_models import CONFIGS, YARN, attention, build, general_delta, write_checkpoint
from tuvutar_models import error, feed_all, make_llm, tokens

TOL = 3e-5
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _g(seed=0):
    return torch.Generator().manual_seed(seed)


# ---- configuration -------------------------------------------------------------------------------------------------
def test_config_reads_every_layer_and_survives_a_round_trip(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    mc = ModelConfig.from_pretrained(path)                 # the ranks come from the tensors' shapes
    again = ModelConfig.from_dict(json.loads(json.dumps(mc.to_dict())))
    for c in (mc, again):
        assert (c.vocab_size, c.hidden_size, c.num_hidden_layers, c.rms_norm_eps, c.embedding_scale, c.postnorm_alpha) == (101, 76, 4, 1e-5, 3.0, 1.7)
        assert (c.is_mla, c.is_hybrid_gdn, c.tie_word_embeddings, c.learned_positions) == (False, True, True, False)
        assert [c.keeps_rows(i) for i in range(4)] == [True, False, True, False] and [c.keeps_state(i) for i in range(4)] == [False, True, False, True]
        assert [c.cache_rank(i) for i in range(4)] == [0, 1, 1, 2] and [c.state_rank(i) for i in range(4)] == [0, 0, 1, 1]
        assert [c.layer_specs[i]["mixer"].get("decay_rank") for i in range(4)] == [None, 5, None, 11]
    from nanoengine_b200.runtime.cache import make_cache_plan
    plan = make_cache_plan(mc, "float32", 64, state_slots=2)
    assert plan.kv_shapes == [(2, 12, 10), (5, 9, 14)] and plan.pools == [7, 23] and plan.delta_shapes == [(3, 10, 10, 1, 0), (2, 18, 18, 1, 0)]
    assert [plan.pooled_rows(l) for l in range(2)] == [16, 8]
    assert plan.kv_block_bytes == 4 * ((64 + 16) * 2 * 22 + (64 + 8) * 5 * 23) and plan.state_slot_bytes == 4 * (3 * 100 + 2 * 324)
    from nanoengine_b200._native import _core as C
    assert plan.plan_bits() == C.PLAN_GQA | C.PLAN_CSA | C.PLAN_GDN
    only = make_cache_plan(ModelConfig.from_dict(CONFIGS["attention_only"]), "float32", 64, state_slots=2)
    assert only.plan_bits() == C.PLAN_GQA | C.PLAN_CSA                       # pooled rows cross pages: no prefix reuse, state or not


@pytest.mark.parametrize("bad", [
    attention(4, 3, 8, 8, 5, 2, 4), attention(4, 2, 8, 8, 0, 2, 4), attention(4, 2, 8, 8, 5, 0, 4), attention(4, 2, 8, 8, 5, 2, 10), attention(4, 2, 8, 8, 5, 2, 3),
    attention(4, 2, 8, 9, 5, 2, 4), general_delta(2, 513, 4), dict(general_delta(4, 8, 8), type="convolution"),
    dict(general_delta(4, 8, 8), mlp={"kind": "experts", "ff": 4})])
def test_config_refuses_what_does_not_fit_together(bad):
    base = {"architecture": "Sapanex", "vocab": 32, "width": 32, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "postln_alpha": 1.0, "layers": [general_delta(4, 8, 8)]}
    ModelConfig.from_dict(base)
    with pytest.raises(ValueError):
        ModelConfig.from_dict({**base, "layers": [bad]})


def test_engine_config_refuses_layouts_it_does_not_run():
    new = lambda: ModelConfig.from_dict(CONFIGS["odd"])
    assert Config(model="x", model_config=new(), max_model_len=200000).model_config.max_position_embeddings == 200000      # no limit of its own
    for bad in (dict(attention_tp=2), dict(kv_cache_dtype="fp8")):
        with pytest.raises(ValueError):
            Config(model="x", model_config=new(), **bad)


# ---- operators against the oracle ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,sc", [(16, 10000.0, YARN), (6, 200000.0, {"factor": 5.0, "original": 2048, "fast": 24.0, "slow": 1.0}), (80, 500.0, YARN),
                                          (2, 100.0, {"factor": 2.0, "original": 7, "fast": 3.0, "slow": 2.9}), (24, 1000.0, None)])
def test_rotary_tables(dims, base, sc):
    freq, factor = oracle.yarn_frequencies(dims, base, sc)
    table = ref.rope_cos_sin_cache(dims, 3000, base, _yarn_of(sc), exact=True)
    a = torch.outer(torch.arange(3000, dtype=torch.float64), torch.tensor(freq, dtype=torch.float64))
    want = torch.cat([a.cos(), a.sin()], -1) * factor
    assert table.dtype == torch.float32 and float((table.double() - want).abs().max()) < 2e-7 * factor
    if sc is not None and dims > 2:
        assert freq != oracle.plain_frequencies(dims, base)


@pytest.mark.parametrize("last", [False, True])
def test_norm_behind_the_sum(last):
    g = _g(4)
    x, y, w, wl = torch.randn(6, 37, generator=g), torch.randn(6, 37, generator=g), torch.randn(37, generator=g), torch.randn(37, generator=g)
    h, x2 = ref.postnorm(y, x, 2.5, w, 1e-2, wl if last else None)
    want = oracle.rms_norm(2.5 * x + y, w, 1e-2)
    assert torch.allclose(x2, want, atol=1e-5) and torch.allclose(h, oracle.rms_norm(want, wl, 1e-2) if last else want, atol=1e-5)
    h, x0 = ref.embed_scaled(torch.tensor([3, 0]), torch.arange(20.0).view(5, 4), 3.0)
    assert torch.equal(x0, 3.0 * torch.arange(20.0).view(5, 4)[[3, 0]]) and torch.equal(h, x0)


def test_activations_of_a_linear():
    x, w = torch.randn(9, 5, generator=_g()), torch.randn(12, 5, generator=_g(1))
    assert torch.allclose(ref.linear(x, w, act="relu2"), oracle.squared_relu(x @ w.T), atol=1e-6)
    got = ref.linear(x, w, act="tanh", act_from=7)
    assert torch.allclose(got, torch.cat([x @ w[:7].T, torch.tanh(x @ w[7:].T)], -1), atol=1e-6)


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("pool", [1, 2, 3, 5, 7, 8, 9, 12, 23, 64, 70, 130])
def test_pooled_rows_have_a_place_of_their_own(pool, page):
    """No two pooled rows share a place, a row's page is there by the time the row is complete, and eight neighbours lie side by side."""
    places = [ref.pooled_row_place(b, pool, page) for b in range(400)]
    assert len(set(places)) == 400 and max(r for _, r in places) < ref.pooled_rows_per_page(pool, page)
    for b, (p, r) in enumerate(places):
        assert p <= (b * pool + pool - 1) // page and (p, r - b % 8) == places[b - b % 8]


def _paged(k, v, pool, page=64):
    """Keys, values and their pooled rows of one sequence in shuffled pages behind rows of another."""
    n = k.shape[0]
    nb = (n + page - 1) // page
    bt = torch.randperm(nb + 2, generator=_g(5))[:nb].int()
    out = []
    for t in (k, v):
        c, p = torch.randn(nb + 2, page, *t.shape[1:], generator=_g(6)), torch.randn(nb + 2, ref.pooled_rows_per_page(pool, page), *t.shape[1:], generator=_g(7))
        for j in range(n):
            c[bt[j // page], j % page] = t[j]
        for b, m in enumerate(oracle.pool_blocks(t, pool)):
            pg, row = ref.pooled_row_place(b, pool, page)
            p[bt[pg], row] = m
        out += [c, p]
    return out[0], out[2], (out[1], out[3]), bt.view(1, -1)


@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 12, 20), (3, 3, 8, 6), (6, 1, 16, 16)])
@pytest.mark.parametrize("window,pool", [(1, 1), (2, 3), (20, 7), (63, 8), (64, 64), (65, 12), (30, 100), (500, 4)])
def test_attention_at_every_edge_of_window_and_blocks(H, G, d, vd, window, pool):
    """One key, or one block, stands out for a query: it counts just inside the window, or just when its block is seen, and not one position further."""
    n = 150
    g = _g(H + window)
    q, k, v = torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, G, vd, generator=g)
    i = n - 1
    seen = max(0, (i - window + 1) // pool)
    for what in ("in", "out", "block", "next block"):
        kk = k.clone()
        j = {"in": i - window + 1, "out": i - window}.get(what)
        b = {"block": seen - 1, "next block": seen}.get(what)
        if j is not None and 0 <= j < i:
            kk[j, 0] = 3.0 * q[i, 0]
        if b is not None and 0 <= b and (b + 1) * pool <= n:
            kk[b * pool: (b + 1) * pool, 0] = 3.0 * q[i, 0]
        want = oracle.window_attention(q, kk, v, 0.4, window, pool)
        kc, vc, pooled, bt = _paged(kk, v, pool)
        for lo in (0, 100, i):
            got = ref.gqa_attention_biased(q[lo:], kc, vc, bt, torch.tensor([0, n - lo]), torch.tensor([n]), 0.4, window, pooled=pooled, pool=pool)
            assert torch.allclose(got.view(n - lo, H, vd), want[lo:], atol=1e-5), (what, lo)
        if what == "block" and b >= 0:                      # it shows: leaving it out changes the result
            off = oracle.window_attention(q, kk, v, 0.4, window, pool, hide=lambda t: ([], [b]))
            assert float((off - want)[i, 0].abs().max()) > 1e-2
    freq = oracle.plain_frequencies(vd, 50.0)
    table = ref.rope_cos_sin_cache(vd, n, 50.0, exact=True)
    got = ref.gqa_attention_biased(q, kc, vc, bt, torch.tensor([0, n]), torch.tensor([n]), 0.4, window, pooled=pooled, pool=pool, turn_back=table)
    assert torch.allclose(got.view(n, H, vd), oracle.rotate(want, freq, back=True), atol=1e-5)


@pytest.mark.parametrize("H,G,d,vd,rot,pool", [(4, 2, 12, 20, 6, 7), (3, 1, 8, 6, 8, 3), (2, 2, 20, 10, 2, 70)])
def test_front_end_statement(H, G, d, vd, rot, pool):
    """Norm over all heads at once, rotations, rows and block means, in portions of any size."""
    n, eps, g = 145, 1e-2, _g(d)
    qkv = torch.randn(n, H * d + G * (d + vd), generator=g)
    qn, kn = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    freq, factor = oracle.yarn_frequencies(rot, 1000.0, YARN)
    kt, vt = ref.rope_cos_sin_cache(rot, n, 1000.0, _yarn_of(YARN), exact=True), ref.rope_cos_sin_cache(vd, n, 1000.0, exact=True)
    q, k, v = qkv.split([H * d, G * d, G * vd], -1)
    want_q = oracle.rotate(oracle.rms_norm(q, qn, eps).view(n, H, d), freq, factor)
    want_k = oracle.rotate(oracle.rms_norm(k, kn, eps).view(n, G, d), freq, factor)
    want_v = oracle.rotate(v.reshape(n, G, vd), oracle.plain_frequencies(vd, 1000.0))
    kc0, vc0, pooled0, bt = _paged(want_k, want_v, pool)
    caches = [torch.full_like(t, 9.0) for t in (kc0, vc0, *pooled0)]
    at = 0
    for m in (1, 2, 60, 1, 1, 5, 58, 17):
        pos = torch.arange(at, at + m)
        got = ref.pooled_attention_prepare(qkv[at: at + m].clone(), H, G, d, vd, qn, kn, eps, pos, kt, vt, *caches, pool, bt[0][pos // 64].long() * 64 + pos % 64, bt,
                                           torch.tensor([0, m]))
        assert torch.allclose(got, want_q[at: at + m], atol=2e-5)
        at += m
    assert at == n
    own = bt[0].long()
    assert all(torch.allclose(a[own].flatten(0, 1)[:n], b[own].flatten(0, 1)[:n], atol=2e-5) for a, b in zip(caches[:2], (kc0, vc0)))
    for b in range(n // pool):
        pg, row = ref.pooled_row_place(b, pool, 64)
        assert all(torch.allclose(a[own[pg], row], w[own[pg], row], atol=2e-5) for a, w in zip(caches[2:], pooled0)), b


@pytest.mark.parametrize("H,d", [(3, 10), (2, 24), (1, 7)])
def test_general_delta_statement(H, d):
    D, n, eps, rank = 32, 21, 1e-3, 6
    cfg = {"vocab": 8, "width": D, "norm": {"eps": eps}, "ranks": [rank], "layers": [general_delta(H, d, rank)]}
    W = oracle.part({k: v.float() for k, v in oracle.random_weights(cfg, 5).items()}, "l0.mix.")
    h = torch.randn(n, D, generator=_g(9))
    proj = torch.cat([h @ W[c].T for c in "rkavg"], -1)
    decay = torch.tanh(h @ W["w1"].T) @ W["w2"].T
    st, outs = torch.randn(3, H, d, d, generator=_g(2)), []              # stale: a fresh sequence ignores it
    for lo, hi in ((0, 9), (9, 10), (10, 12), (12, n)):
        outs.append(ref.general_delta(proj[lo:hi], decay[lo:hi], W["w0"], W["a.b"], W["norm"], st, torch.tensor([1]), torch.tensor([0, hi - lo]),
                                      torch.tensor([int(lo == 0)]), H, d, d, eps))
    Wd = {k: v.double() for k, v in W.items()}
    want = oracle.general_delta(h.double(), Wd, {"heads": H, "dim": d}, eps)
    assert torch.allclose(torch.cat(outs) @ W["o"].T, want.float(), atol=2e-5)


# ---- the engine ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_single_tokens_agree_with_the_oracle(name, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=2.0)
    toks = tokens(150, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", "cpu", pages=4)
    for cuts in ([150], [2], [1], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64], [129, 1]):
        assert error(feed_all(llm, None, toks, cuts), want) < TOL, cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 4 and llm.engine.scheduler.num_fed() == 0


def test_layers_one_by_one(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    toks, trace = tokens(90, cfg["vocab"], 6), []
    llm = make_llm(path, "float32", "cpu", pages=4)
    model = llm.engine.executor.runner.model
    model.trace_residual = []
    oracle.forward(cfg, W, toks, trace)
    feed_all(llm, None, toks, [90])
    assert len(model.trace_residual) == len(trace) == 5
    for got, want in zip(model.trace_residual, trace):
        assert float((got.double() - want).abs().max()) < 1e-4


def test_single_keys_and_blocks_show_in_the_logits(tmp_path):
    """Queries scaled until single keys stand out: hiding a token or a block from the oracle changes the logits, and so does a window or a pool of
    another size; the engine agrees with the oracle - in one prompt and token by token."""
    cfg, W, path = build("aligned", tmp_path, sharp=2.0)
    toks = tokens(140, cfg["vocab"], 4)
    want = oracle.forward(cfg, W, toks)
    for key in (0, 63, 64, 127):
        assert error(oracle.forward(cfg, W, toks, hide=lambda i: ([key], [])), want) > 100 * TOL, key
    for block in (0, 1, 15, 16):
        assert error(oracle.forward(cfg, W, toks, hide=lambda i: ([], [block])), want) > 10 * TOL, block
    for field in ("size", "pool"):
        for off in (-1, 1):
            other = json.loads(json.dumps(cfg))
            for L in other["layers"]:
                if L["type"] == "attention":
                    L["mixer"]["mask"][field] += off
            assert error(oracle.forward(other, W, toks), want) > 20 * TOL, (field, off)
    llm = make_llm(path, "float32", "cpu", pages=4)
    assert error(feed_all(llm, None, toks, [140]), want) < TOL
    assert error(feed_all(llm, None, toks, [100, 1]), want) < TOL


def test_other_page_sizes(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    toks = tokens(100, cfg["vocab"], 5)
    want = oracle.forward(cfg, W, toks)
    for page, pages in ((16, 8), (128, 2)):
        llm = LLM(Config(model=path, dtype="float32", device="cpu", max_num_seqs=2, num_kvcache_blocks=pages, kvcache_block_size=page, max_model_len=128,
                         max_num_batched_tokens=128, enable_prefix_caching=False, executor_backend="inproc", status_log_interval_s=0))
        assert error(feed_all(llm, None, toks, [37, 1, 2, 20]), want) < TOL, page


def test_bfloat16_stays_near_the_oracle(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    toks = tokens(90, cfg["vocab"], 2)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "bfloat16", "cpu", pages=4)
    assert error(feed_all(llm, None, toks, [50, 1, 9]), want) < 0.08


def test_mixed_batches_with_pages_and_slots_used_again(tmp_path):
    cfg, W, path = build("odd", tmp_path, sharp=2.0)
    reqs = {i: tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate([130, 70, 3, 1, 66, 65, 40, 129])}
    want = {i: oracle.forward(cfg, W, t) for i, t in reqs.items()}
    llm = make_llm(path, "float32", "cpu", pages=6, slots=4)
    at, live, todo, got, ids = {}, [], list(reqs), {i: [] for i in reqs}, {}
    rng = np.random.default_rng(0)
    held = lambda: sum((len(reqs[i]) + 63) // 64 for i in live)
    step = 0
    while todo or live:
        while todo and len(live) < 4 and held() + (len(reqs[todo[0]]) + 63) // 64 <= 6:
            i = todo.pop(0)
            live.append(i); at[i] = 0; ids[i] = 100 + step * 10 + i
        entries, wants, who = [], [], []
        for i in live:
            if rng.random() < 0.2:
                continue                                                # left out of this step
            n = int(rng.choice([1, 1, 2, 3, 17, 64]))
            part = reqs[i][at[i]: at[i] + n]
            entries.append((ids[i], part)); wants.append(list(range(len(part)))); who.append(i)
        if not entries:
            continue
        out = llm.feed(entries, wants)
        row = 0
        for i, (_, part) in zip(who, entries):
            got[i].append(torch.from_numpy(out[row: row + len(part)])); row += len(part)
            at[i] += len(part)
            if at[i] == len(reqs[i]):
                llm.end_feed([ids[i]]); live.remove(i)
        step += 1
    for i in reqs:
        assert error(torch.cat(got[i]), want[i]) < TOL, i
    assert llm.engine.scheduler.num_free_blocks(0) == 6 and llm.engine.scheduler.num_free_state_slots(0) == 4


@pytest.mark.parametrize("name", ["aligned", "attention_only"])
def test_greedy_generation_through_the_scheduler(name, tmp_path):
    cfg, W, path = build(name, tmp_path)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (70, 2, 33, 1, 64)]
    want = [oracle.greedy(cfg, W, p, 5) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    for kw in (dict(), dict(max_num_batched_tokens=16), dict(max_num_batched_tokens=65)):       # chunked prompts, cut anywhere
        llm = make_llm(path, "float32", "cpu", pages=9, **kw)
        outs = {o["seq_id"]: o["token_ids"] for o in llm.generate(prompts, sp)}
        assert [outs[i + 1] for i in range(len(prompts))] == want, kw


def test_equal_prompts_share_no_pages(tmp_path):
    """Pooled rows of a page cover tokens of later pages, so a prefix is never reused, with or without recurrent layers."""
    cfg, W, path = build("attention_only", tmp_path)
    llm = LLM(Config(model=path, dtype="float32", device="cpu", max_num_seqs=4, num_kvcache_blocks=12, max_model_len=256, enable_prefix_caching=True,
                     executor_backend="inproc", status_log_interval_s=0))
    base = tokens(128, cfg["vocab"], 1)
    sp = SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True)
    for tail in (2, 3):
        p = base + tokens(10, cfg["vocab"], tail)
        assert llm.generate([p], sp)[0]["token_ids"] == oracle.greedy(cfg, W, p, 3)


def test_preempted_sequences_recompute_or_come_back_from_the_host(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    prompts = [tokens(60, cfg["vocab"], 40 + i) for i in range(3)]
    want = [oracle.greedy(cfg, W, p, 8) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    for host in (0, 8):
        llm = make_llm(path, "float32", "cpu", pages=4, num_host_kvcache_blocks=host)
        ids = [llm.add_request(p, sp) for p in prompts]
        acc, pre = {}, 0
        for _ in range(400):
            if llm.is_finished():
                break
            for so in llm.step():
                acc.setdefault(so.seq_id, []).extend(so.token_ids)
            pre += sum(llm.engine.scheduler.get(i).num_preemptions for i in ids if llm.engine.scheduler.get(i) is not None)
        assert pre > 0 and [acc[i] for i in ids] == want


@pytest.mark.parametrize("transport", ["copy", "push"])
def test_cache_families_and_migration_between_engines(tmp_path, transport):
    """Keys, values, pooled rows and states of every layer move with a sequence (prefill engine -> decode engine)."""
    from nanoengine_b200.parallel.kv_transfer import KVMigrator, LocalTransport, connect_inproc
    cfg, W, path = build("aligned", tmp_path)
    pre, dec = make_llm(path, "float32", "cpu", pages=9, mode="prefill", engine_id="p"), make_llm(path, "float32", "cpu", pages=9, mode="decode", engine_id="d")
    kv = dec.engine.executor.runner.cache
    assert [f["name"] for f in kv.page_families()] == [f"{n}_{i}" for i in range(3) for n in ("key", "value", "pooled_key", "pooled_value")]
    assert [f["name"] for f in kv.slot_families()] == ["delta_state_0", "delta_state_1"]
    assert kv.plan.state_slot_bytes == sum(f["slot_bytes"] for f in kv.slot_families()) and kv.plan.block_bytes == sum(f["page_bytes"] for f in kv.page_families())
    assert sum(t.numel() * t.element_size() for t in kv.block_views(2)) == kv.plan.block_bytes
    prompt = tokens(75, cfg["vocab"], 9)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    blobs = pre.generate([prompt], sp, return_serialized=True)
    if transport == "copy":
        tr = LocalTransport([pre.engine.executor.runner], [dec.engine.executor.runner])
        dec.engine.migrator = KVMigrator(tr, dec.engine.engine_info(), pre.engine.engine_info())
    else:
        connect_inproc(pre.engine, dec.engine)
    for b in blobs:
        dec.add_request_payload(b)
    out = dec.generate()
    assert out[0]["token_ids"][-5:] == oracle.greedy(cfg, W, prompt, 6)[1:]


def test_random_weights_cover_the_checkpoint_and_loading_is_strict(tmp_path):
    llm = LLM(Config(model="tiny-sapanex", device="cpu", dtype="float32", num_kvcache_blocks=8, max_model_len=256, max_num_seqs=4))
    outs = llm.generate([[1, 2, 3, 4]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(outs[0]["token_ids"]) == 4
    assert PRESETS["sapanex-7b"]().num_hidden_layers == 32
    cfg, W, _ = build("odd", tmp_path)
    for change in (lambda w: w.pop("l1.mix.a.b"), lambda w: w.pop("l1.mix.w1"), lambda w: w.pop("l0.mix.v"), lambda w: w.update(extra=torch.zeros(2))):
        w = dict(W)
        change(w)
        with pytest.raises(ValueError):
            make_llm(write_checkpoint(os.path.join(str(tmp_path), "bad"), cfg, w), "float32", "cpu", pages=4)


def test_weights_can_be_replaced_in_place(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    W2 = oracle.random_weights(cfg, 77)
    llm = make_llm(path, "float32", "cpu", pages=4)
    llm.update_weights(list(W2.items()))
    toks = tokens(20, cfg["vocab"], 3)
    assert error(feed_all(llm, None, toks, [20]), oracle.forward(cfg, W2, toks)) < TOL


def test_replay_program(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(66, cfg["vocab"], 1), tokens(5, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:], "want": [3]}, {"id": "a", "tokens": a[64:65], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[65:], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [4]}], "end": ["b"]}]
    r = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "192",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    wa, wb = oracle.forward(cfg, W, a), oracle.forward(cfg, W, b)
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    assert error(read(0), wa[[0, 63]]) < TOL and error(read(1), torch.stack([wb[4], wa[64]])) < TOL and error(read(3), wb[4:5]) < TOL
    assert not (out / "2.f32").exists()
