"""Gipozen on CPU: the reader of its configuration, every operator's PyTorch statement against the plain oracle, and the engine - scheduler, pages,
windows of the convolutions, portions, mixed batches, generation - in 32-bit against the oracle's logits."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gipozen_oracle as oracle
from gipozen_models import CONFIGS, attention, build, dense, moe, write_checkpoint
from nanoengine_b200 import Config, LLM, SamplingParams
from nanoengine_b200.models.config import PRESETS, ModelConfig
from nanoengine_b200.ops import reference as ref
from tuvutar_models import error, feed_all, make_llm, tokens

TOL = 3e-5
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _g(seed=0):
    return torch.Generator().manual_seed(seed)


# ---- configuration -------------------------------------------------------------------------------------------------
def test_config_reads_every_layer_and_survives_a_round_trip(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    mc = ModelConfig.from_pretrained(path)
    again = ModelConfig.from_dict(json.loads(json.dumps(mc.to_dict())))
    for c in (mc, again):
        assert (c.vocab_size, c.hidden_size, c.num_hidden_layers, c.rms_norm_eps, c.logit_scale) == (101, 76, 4, 1e-5, 0.7)
        assert (c.is_mla, c.is_hybrid_gdn, c.tie_word_embeddings, c.learned_positions) == (False, True, False, False)
        assert [c.kv_source_layer(i) for i in range(4)] == [0, 0, 2, 0] and [c.keeps_rows(i) for i in range(4)] == [True, False, True, False]
        assert [c.cache_rank(c.kv_source_layer(i)) for i in range(4)] == [0, 0, 1, 0] and [c.state_rank(i) for i in range(4)] == [0, 1, 2, 3]
    from nanoengine_b200._native import _core as C
    from nanoengine_b200.runtime.cache import make_cache_plan
    plan = make_cache_plan(mc, "float32", 64, state_slots=2)
    assert plan.kv_shapes == [(2, 22, 10), (3, 18, 14)]
    assert plan.delta_shapes == [(0, 0, 0, 4, 132 + 64), (0, 0, 0, 3, 132), (0, 0, 0, 2, 54 + 96), (0, 0, 0, 5, 176)]
    assert plan.kv_block_bytes == 4 * 64 * (2 * 32 + 3 * 32) and plan.state_slot_bytes == 4 * (3 * 196 + 2 * 132 + 150 + 4 * 176)
    assert plan.plan_bits() == C.PLAN_GQA | C.PLAN_GDN
    only = make_cache_plan(ModelConfig.from_dict(CONFIGS["stateless"]), "float32", 64, state_slots=2)
    assert only.plan_bits() == C.PLAN_GQA and not only.needs_state_slots
    some = ModelConfig.from_dict(CONFIGS["fine"])                       # layers with a single tap have no window
    assert [some.keeps_state(i) for i in range(4)] == [False, True, True, False] and some.is_hybrid_gdn


@pytest.mark.parametrize("bad", [
    attention(4, 3, 8, 8, 5, 2, 4, 0.1), attention(4, 2, 8, 8, 0, 2, 4, 0.1), attention(4, 2, 8, 8, 5, -1, 4, 0.1), attention(4, 2, 8, 8, 5, 2, 17, 0.1),
    attention(4, 2, 8, 8, 5, 2, 4, 0.1, src=1), attention(4, 4, 8, 8, 5, 2, 4, 0.1, src=0), attention(4, 2, 8, 16, 5, 2, 4, 0.1, src=0),
    attention(4, 2, 8, 8, 5, 2, 4, 0.1, moe(4, 0, 5, 8, 0, 1.0)), attention(4, 2, 8, 8, 5, 2, 4, 0.1, moe(4, 0, 2, 8, 0, 0.0)),
    attention(4, 2, 8, 8, 5, 2, 4, 0.1, moe(4, 0, 2, 8, 8, 1.0, -1.0)), dict(attention(4, 2, 8, 8, 5, 2, 4, 0.1), type="delta"),
    attention(4, 2, 8, 8, 5, 2, 4, 0.1, {"kind": "other", "ff": 4})])
def test_config_refuses_what_does_not_fit_together(bad):
    first = attention(4, 2, 8, 8, 5, 2, 4, 0.1)
    base = {"architecture": "Gipozen", "vocab": 32, "width": 32, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "layers": [first, attention(4, 2, 8, 8, 9, 0, 2, 0.2, src=0)]}
    ModelConfig.from_dict(base)
    with pytest.raises(ValueError):
        ModelConfig.from_dict({**base, "layers": [first, bad]})


def test_a_reader_of_a_reader_is_refused():
    layers = [attention(4, 2, 8, 8, 5, 2, 4, 0.1), attention(4, 2, 8, 8, 5, 2, 4, 0.1, src=0), attention(4, 2, 8, 8, 5, 2, 4, 0.1, src=1)]
    with pytest.raises(ValueError):
        ModelConfig.from_dict({"architecture": "Gipozen", "vocab": 32, "width": 32, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "layers": layers})


def test_engine_config_refuses_layouts_it_does_not_run():
    new = lambda: ModelConfig.from_dict(CONFIGS["odd"])
    assert Config(model="x", model_config=new(), max_model_len=200000).max_model_len == 200000      # no limit of its own
    for bad in (dict(attention_tp=2), dict(kv_cache_dtype="fp8"), dict(attention_dp=2, ffn_ep=2)):
        with pytest.raises(ValueError):
            Config(model="x", model_config=new(), **bad)


# ---- operators against the oracle ------------------------------------------------------------------------------------
def test_depth_average():
    g = _g(4)
    table, ids, n1 = torch.randn(9, 21, generator=g), torch.tensor([3, 0, 8]), torch.tensor([0.7])
    h, x, bank = ref.depth_embed(ids, table, n1, 1e-2, 4)
    assert bank.shape == (4, 3, 21) and torch.equal(x, table[ids]) and torch.allclose(h, oracle.rms_norm(table[ids], 0.7, 1e-2), atol=1e-6)
    history = [x]
    for i in range(3):
        y, w = torch.randn(3, 21, generator=g), torch.randn(i + 2, generator=g)
        h, mid = ref.depth_mix(y, x, n1, 1e-2)
        assert torch.allclose(mid, x + y) and torch.allclose(h, oracle.rms_norm(x + y, 0.7, 1e-2), atol=1e-6)
        z = torch.randn(3, 21, generator=g)
        h, x = ref.depth_mix(z, mid, n1, 1e-2, bank, i + 1, w)
        history.append(mid + z)
        want = oracle.depth_average(history, w)
        assert torch.allclose(x, want, atol=1e-5) and torch.allclose(h, oracle.rms_norm(want, 0.7, 1e-2), atol=1e-5)


def test_normed_powers():
    z, coef = 2 * torch.randn(7, 13, generator=_g()), torch.tensor([1.1, -0.4, 0.3, 0.2])
    assert torch.allclose(ref.poly_norm(z, coef, 1e-2), oracle.poly_norm(z, coef, 1e-2), atol=1e-5)


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("taps", [1, 2, 3, 6])
def test_short_convolution_in_portions(taps, page):
    n, qw, G, kd, vd = 83, 12, 2, 5, 3
    C = qw + G * (kd + vd)
    g = _g(taps)
    u, w = torch.randn(n, C + 4, generator=g), torch.randn(C, taps, generator=g)
    want = oracle.short_conv(u[:, :C], w)
    nb = (n + page - 1) // page
    bt = torch.randperm(nb + 1, generator=g)[:nb]
    kc, vc = torch.full((nb + 1, page, G, kd), 9.0), torch.full((nb + 1, page, G, vd), 9.0)
    win, slots = torch.randn(3, taps - 1, C, generator=g), torch.tensor([1])          # stale: a fresh sequence ignores it
    at, out = 0, []
    for m in (1, 2, 40, 1, 1, 30, 3, 5):
        pos = torch.arange(at, at + m)
        rows = bt[pos // page] * page + pos % page
        out.append(ref.conv_rows(u[at: at + m], w.t().contiguous(), qw, kc, vc, rows, win if taps > 1 else None, slots, torch.tensor([0, m]), torch.tensor([int(at == 0)])))
        at += m
    assert at == n and torch.allclose(torch.cat(out), want[:, :qw], atol=1e-5)
    assert torch.allclose(kc[bt].flatten(0, 1)[:n].flatten(1), want[:, qw: qw + G * kd], atol=1e-5)
    assert torch.allclose(vc[bt].flatten(0, 1)[:n].flatten(1), want[:, qw + G * kd:], atol=1e-5)


def paged(k, v, page=64):
    """Keys and values of one sequence in shuffled pages behind rows of another."""
    n = k.shape[0]
    nb = (n + page - 1) // page
    bt = torch.randperm(nb + 2, generator=_g(5))[:nb].int()
    out = []
    for t in (k, v):
        c = torch.randn(nb + 2, page, *t.shape[1:], generator=_g(6))
        for j in range(n):
            c[bt[j // page], j % page] = t[j]
        out.append(c)
    return (*out, bt.view(1, -1))


def plain_attention(q, k, v, scale, size, keep, lam, diff, eps, gate, hide=None):
    """q [n, H, 2, d], k [n, G, 2 d], v [n, G, dv] -> [n, H dv]"""
    n, H, G, d = q.shape[0], q.shape[1], k.shape[1], q.shape[3]
    heads = []
    for x in range(H):
        y = x // (H // G)
        a1, a2 = (oracle.one_map(q[:, x, i], k[:, y, i * d: (i + 1) * d], v[:, y], scale, size, keep, hide) for i in (0, 1))
        heads.append(oracle.combine(a1, a2, lam, diff, eps))
    return torch.cat(heads, -1) * oracle.sigmoid(gate)


@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 12, 20), (3, 3, 8, 6), (6, 1, 16, 16)])
@pytest.mark.parametrize("size,keep", [(1, 0), (1, 1), (2, 3), (20, 0), (20, 7), (63, 1), (64, 64), (65, 70), (30, 100), (500, 4)])
def test_attention_at_every_edge_of_window_and_kept_tokens(H, G, d, vd, size, keep):
    """One key of one map stands out for a query: it counts just inside the window, or among the kept tokens, and not one position further."""
    n = 150
    g = _g(H + size)
    q, k, v = torch.randn(n, H, 2, d, generator=g), torch.randn(n, G, 2 * d, generator=g), torch.randn(n, G, vd, generator=g)
    gate, lam, diff, eps = torch.randn(n, H * vd, generator=g), 0.45, 0.3, 1e-3
    i = n - 1
    for m, j in ((0, i - size + 1), (1, i - size), (0, keep - 1), (1, keep)):
        if not 0 <= j < i:
            continue
        kk = k.clone()
        kk[j, 0, m * d: (m + 1) * d] = 3.0 * q[i, 0, m]
        want = plain_attention(q, kk, v, 0.4, size, keep, lam, diff, eps, gate)
        kc, vc, bt = paged(kk, v)
        for lo in (0, 100, i):
            got = ref.differential_attention(q[lo:], kc, vc, bt, torch.tensor([0, n - lo]), torch.tensor([n]), 0.4, size, keep, torch.tensor([lam]), 1 - diff, eps, gate[lo:])
            assert torch.allclose(got, want[lo:], atol=2e-5), (m, j, lo)
        if i - j < size or j < keep:                        # it shows: leaving it out changes the result
            off = plain_attention(q, kk, v, 0.4, size, keep, lam, diff, eps, gate, hide=lambda t: [j])
            assert float((off - want)[i].abs().max()) > 1e-2


def test_attention_without_a_window_sees_everything():
    n, g = 90, _g(3)
    q, k, v, gate = torch.randn(n, 2, 2, 8, generator=g), torch.randn(n, 1, 16, generator=g), torch.randn(n, 1, 12, generator=g), torch.randn(n, 24, generator=g)
    kc, vc, bt = paged(k, v)
    got = ref.differential_attention(q, kc, vc, bt, torch.tensor([0, n]), torch.tensor([n]), 0.4, 0, 0, torch.tensor([0.3]), 0.6, 1e-4, gate)
    assert torch.allclose(got, plain_attention(q, k, v, 0.4, n, 0, 0.3, 0.4, 1e-4, gate), atol=2e-5)


def test_mixing_factor():
    from nanoengine_b200.models.mixers import DifferentialAttentionMixer
    cfg = CONFIGS["aligned"]
    W = oracle.part(oracle.random_weights(cfg, 5), "l0.mix.")
    m = DifferentialAttentionMixer(128, 8, 2, 32, 48, 1.0, 40, 5, 0.25, 4, 1e-6, 0, False, 0, torch.float32, "cpu")
    m.load({k: v.float() for k, v in W.items()})
    want = oracle.mixing_factor(W, 0.25)
    assert abs(float(m.mixing) - want) < 1e-6 and abs(want - 0.25) > 1e-2


@pytest.mark.parametrize("identity,top,shared", [(0, 1, 0), (3, 2, 0), (2, 5, 24), (4, 8, 40)])
def test_mixture(identity, top, shared):
    from nanoengine_b200.models.layers import GatedSharedMoE
    D, E, F, n = 24, 6, 20, 40
    spec = moe(E, identity, top, F, shared, 0.7, 0.4)
    cfg = {"vocab": 8, "width": D, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "layers": [attention(2, 1, 8, 8, 4, 0, 1, 0.1, spec)]}
    W = oracle.part({k: v.float() for k, v in oracle.random_weights(cfg, 7).items()}, "l0.mlp.")
    M = GatedSharedMoE(D, E, identity, top, F, ("clamp_linear", 0.7, oracle.SLOPE), shared, ("clamp_linear", 0.4, oracle.SLOPE) if shared else None, torch.float32, "cpu")
    M.router_weight[: E + identity].copy_(W["router"])
    M.correction.copy_(W["correction"])
    for e in range(E):
        for which in ("gate", "up", "down"):
            M.experts.load_expert(e, which, W[f"e{e}.{which}"])
    if shared:
        M.router_weight[E + identity:].copy_(W["shared.sg"])
        M.shared.gate_up_proj.set_weight(torch.cat([W["shared.gate"], W["shared.up"]], 0))
        M.shared.down_proj.set_weight(W["shared.down"])
    h = 1.5 * torch.randn(n, D, generator=_g(9))
    want = oracle.experts(h.double(), {k: v.double() for k, v in W.items()}, spec)
    assert torch.allclose(M(h), want.float(), atol=2e-5)
    if identity and top < E:
        chosen = [oracle.route(z, W["correction"], top)[0] for z in h @ W["router"].T]
        plain = [oracle.route(z, torch.zeros(E + identity), top)[0] for z in h @ W["router"].T]
        assert any(i >= E for c in chosen for i in c) and chosen != plain            # identity experts are chosen, the correction decides some choices


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
    assert len(model.trace_residual) == len(trace) == 4
    for got, want in zip(model.trace_residual, trace):
        assert float((got.double() - want).abs().max()) < 1e-4


def test_single_keys_and_every_part_show_in_the_logits(tmp_path):
    """Hiding a key from the oracle changes the logits, and so does a window, a number of kept tokens, or a tensor of another value; the engine agrees
    with the oracle - in one prompt and token by token."""
    cfg, W, path = build("aligned", tmp_path, sharp=2.0)
    toks = tokens(140, cfg["vocab"], 4)
    want = oracle.forward(cfg, W, toks)
    for key in (0, 4, 63, 64, 127):
        assert error(oracle.forward(cfg, W, toks, hide=lambda i: [key]), want) > 100 * TOL, key
    for field in ("size", "keep_first"):
        for off in (-1, 1):
            other = json.loads(json.dumps(cfg))
            for L in other["layers"]:
                L["mixer"]["mask"][field] += off
            assert error(oracle.forward(other, W, toks), want) > 20 * TOL, (field, off)
    for name in ("l0.dwa", "l2.mix.lq2", "l0.mlp.act", "l1.mlp.correction", "l1.mlp.shared.sg", "l2.mix.q.conv", "l0.mix.v.conv", "l1.norm2", "final.norm"):
        W2 = dict(W, **{name: W[name] * 1.5 if W[name].dim() == 0 else W[name].flip(0) + 0.1})
        assert error(oracle.forward(cfg, W2, toks), want) > 20 * TOL, name
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
    assert error(feed_all(llm, None, toks, [50, 1, 9]), want) < 0.15


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


@pytest.mark.parametrize("name", ["aligned", "stateless"])
def test_greedy_generation_through_the_scheduler(name, tmp_path):
    cfg, W, path = build(name, tmp_path)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (70, 2, 33, 1, 64)]
    want = [oracle.greedy(cfg, W, p, 5) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    for kw in (dict(), dict(max_num_batched_tokens=16), dict(max_num_batched_tokens=65)):       # chunked prompts, cut anywhere
        llm = make_llm(path, "float32", "cpu", pages=9, **kw)
        outs = {o["seq_id"]: o["token_ids"] for o in llm.generate(prompts, sp)}
        assert [outs[i + 1] for i in range(len(prompts))] == want, kw


@pytest.mark.parametrize("name,shared", [("aligned", False), ("stateless", True)])
def test_equal_prefixes_share_pages_only_without_convolutions(name, shared, tmp_path):
    """A prefix's pages hold everything a sequence needs unless its convolutions carry a window."""
    cfg, W, path = build(name, tmp_path)
    llm = LLM(Config(model=path, dtype="float32", device="cpu", max_num_seqs=4, num_kvcache_blocks=12, max_model_len=256, enable_prefix_caching=True,
                     executor_backend="inproc", status_log_interval_s=0))
    base = tokens(128, cfg["vocab"], 1)
    sp = SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True)
    for tail in (2, 3):
        p = base + tokens(10, cfg["vocab"], tail)
        assert llm.generate([p], sp)[0]["token_ids"] == oracle.greedy(cfg, W, p, 3)
    assert (llm.engine.scheduler.metrics_summary()["prompt_tokens"] < 2 * 138) == shared


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
    """Keys, values and convolution windows of every layer move with a sequence (prefill engine -> decode engine)."""
    from nanoengine_b200.parallel.kv_transfer import KVMigrator, LocalTransport, connect_inproc
    cfg, W, path = build("aligned", tmp_path)
    pre, dec = make_llm(path, "float32", "cpu", pages=9, mode="prefill", engine_id="p"), make_llm(path, "float32", "cpu", pages=9, mode="decode", engine_id="d")
    kv = dec.engine.executor.runner.cache
    assert [f["name"] for f in kv.page_families()] == [f"{n}_{i}" for i in range(3) for n in ("key", "value")]
    assert [f["name"] for f in kv.slot_families()] == [f"delta_conv_{i}" for i in range(4)]
    assert kv.plan.state_slot_bytes == sum(f["slot_bytes"] for f in kv.slot_families()) and kv.plan.block_bytes == sum(f["page_bytes"] for f in kv.page_families())
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
    llm = LLM(Config(model="tiny-gipozen", device="cpu", dtype="float32", num_kvcache_blocks=8, max_model_len=256, max_num_seqs=4))
    outs = llm.generate([[1, 2, 3, 4]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(outs[0]["token_ids"]) == 4
    assert PRESETS["gipozen-7b"]().num_hidden_layers == 24
    cfg, W, _ = build("odd", tmp_path)
    for change in (lambda w: w.pop("l1.mix.lq1"), lambda w: w.pop("l1.mlp.e4.up"), lambda w: w.pop("l0.mix.v.conv"), lambda w: w.pop("l3.dwa"),
                   lambda w: w.update({"l1.mix.k": torch.zeros(2)})):
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
