"""Filasun on CPU: the reader of its configuration, every operator's PyTorch statement against the plain oracle, and the engine - scheduler,
pages, state slots, portions, mixed batches, generation - in 32-bit against the oracle's logits."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import filasun_oracle as oracle
from filasun_models import CONFIGS, build, mamba2, parallel, write_checkpoint
from nanoengine_b200 import Config, LLM, SamplingParams
from nanoengine_b200.models.config import PRESETS, ModelConfig
from nanoengine_b200.ops import reference as ref
from tuvutar_models import error, feed_all, make_llm, tokens

TOL = 3e-5
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- configuration -------------------------------------------------------------------------------------------------
def test_config_reads_every_layer_and_survives_a_round_trip():
    mc = ModelConfig.from_dict(CONFIGS["odd"])
    again = ModelConfig.from_dict(json.loads(json.dumps(mc.to_dict())))
    for c in (mc, again):
        assert (c.vocab_size, c.hidden_size, c.num_hidden_layers, c.rms_norm_eps, c.hc_mult, c.final_logit_softcapping) == (97, 76, 4, 1e-5, 3, 9.0)
        assert (c.max_position_embeddings, c.learned_positions, c.is_mla, c.is_hybrid_gdn) == (400, True, False, True)
        assert [c.keeps_rows(i) for i in range(4)] == [True, False, True, False] and all(c.keeps_state(i) for i in range(4))
        assert [c.cache_rank(i) for i in range(4)] == [0, 1, 1, 2] and [c.state_rank(i) for i in range(4)] == [0, 1, 2, 3]
    from nanoengine_b200.runtime.cache import make_cache_plan
    plan = make_cache_plan(mc, "float32", 64, state_slots=2)
    assert plan.kv_shapes == [(2, 12, 20), (5, 9, 7)] and plan.delta_shapes == [(3, 14, 10, 1, 0), (6, 10, 14, 3, 144), (2, 5, 17, 1, 0), (3, 18, 36, 2, 126)]
    assert plan.kv_block_bytes == 64 * 4 * (2 * 32 + 5 * 16) and plan.state_slot_bytes == 4 * (3 * 140 + 6 * 140 + 2 * 144 + 2 * 85 + 3 * 648 + 126)


@pytest.mark.parametrize("bad", [
    dict(layers=[mamba2(4, 8, 8, groups=3)]), dict(layers=[mamba2(4, 8, 8, norm_groups=5)]), dict(layers=[mamba2(4, 8, 8, conv=0)]),
    dict(layers=[parallel(4, 3, 8, 8, 5, 2, 8, 8)]), dict(layers=[parallel(4, 2, 8, 8, 0, 2, 8, 8)]), dict(layers=[parallel(4, 2, 8, 8, 5, 2, 8, 8, decay=[0.5])]),
    dict(layers=[parallel(4, 2, 8, 8, 5, 2, 8, 8, softcap=-1.0)]), dict(layers=[dict(mamba2(4, 8, 8), type="convolution")]), dict(streams=0), dict(logit_softcap=0.0),
    dict(layers=[dict(mamba2(4, 8, 8), mlp={"kind": "experts", "ff": 4, "limit": 1.0})])])
def test_config_refuses_what_does_not_fit_together(bad):
    base = {"architecture": "Filasun", "vocab": 32, "width": 32, "norm": {"eps": 1e-6}, "streams": 2, "logit_softcap": 5.0, "max_positions": 64, "layers": [mamba2(4, 8, 8)]}
    ModelConfig.from_dict(base)
    with pytest.raises(ValueError):
        ModelConfig.from_dict({**base, **bad})


def test_engine_config_keeps_to_the_learned_positions_and_refuses_layouts():
    new = lambda: ModelConfig.from_dict(CONFIGS["odd"])
    assert Config(model="x", model_config=new()).max_model_len == 400
    for bad in (dict(max_model_len=401), dict(attention_tp=2), dict(kv_cache_dtype="fp8")):
        with pytest.raises(ValueError):
            Config(model="x", model_config=new(), **bad)


# ---- operators against the oracle ------------------------------------------------------------------------------------
def _g(seed=0):
    return torch.Generator().manual_seed(seed)


@pytest.mark.parametrize("S", [1, 2, 5])
def test_streams(S):
    g = _g(S)
    x, y = torch.randn(6, S, 37, generator=g), torch.randn(6, 37, generator=g)
    wi, wo, mix, wn = torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g), torch.randn(37, generator=g)
    h, x2 = ref.stream_mix(y, x, wo, mix, wi, wn, 1e-2)
    want = oracle.streams_write(x, y, wo, mix)
    assert torch.allclose(x2, want, atol=1e-5) and torch.allclose(h, oracle.rms_norm(oracle.streams_read(want, wi), wn, 1e-2), atol=1e-4)
    if S > 1:                                   # from / to matters
        assert not torch.allclose(x2, oracle.streams_write(x, y, wo, mix.T), atol=1e-2)
    table, pos = torch.randn(9, 37, generator=g), torch.randn(20, 37, generator=g)
    h, x0 = ref.stream_embed(torch.tensor([3, 0]), torch.tensor([0, 17]), table, pos, wi, wn, 1e-2)
    e = table[[3, 0]] + pos[[0, 17]]
    assert torch.equal(x0, e[:, None].repeat(1, S, 1)) and torch.allclose(h, oracle.rms_norm(e * wi.sum(), wn, 1e-2), atol=1e-4)


def test_clamped_feed_forward_and_caps():
    W = {"p.gate": torch.randn(12, 5, generator=_g()).double() * 2, "p.up": torch.randn(12, 5, generator=_g(1)).double() * 2, "p.down": torch.eye(12).double()}
    h = torch.randn(30, 5, generator=_g(2)).double()
    gu = torch.cat([h @ W["p.gate"].T, h @ W["p.up"].T], -1)
    got = ref.glu_act(*gu.chunk(2, -1), ("clamp_linear", 1.4, 1.702))
    assert torch.allclose(got, oracle.clamped_ff(h, W, "p.", 1.4), atol=1e-9)
    assert float((gu.abs() > 1.4).float().mean()) > 0.3
    assert torch.allclose(ref.cap_logits(gu, 2.5), oracle.cap(gu, 2.5))


def _paged(k, v, page=64, stale=None):
    """Keys and values of one sequence in shuffled pages behind rows of another."""
    n = k.shape[0]
    nb = (n + page - 1) // page
    bt = torch.randperm(nb + 2, generator=_g(5))[:nb].int()
    caches = []
    for t in (k, v):
        c = torch.randn(nb + 2, page, *t.shape[1:], generator=_g(6))
        for j in range(n):
            c[bt[j // page], j % page] = t[j]
        caches.append(c)
    return caches[0], caches[1], bt.view(1, -1)


@pytest.mark.parametrize("H,G,d,vd", [(4, 2, 12, 20), (3, 3, 8, 5), (6, 1, 16, 16)])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 130, 500])
def test_windowed_attention_at_every_edge(H, G, d, vd, window):
    """One key stands out for the last query: it counts inside the window, also as its last key, and not a position further out."""
    n = 150
    g = _g(H + window)
    q, k, v = torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, G, vd, generator=g)
    for dist in (window - 1, window, 1, 149):
        kk = k.clone()
        j = n - 1 - dist
        if 0 <= j < n - 1:
            kk[j, 0] = 3.0 * q[n - 1, 0]
        want = oracle.window_attention(q, kk, v, 0.4, 30.0, window)
        kc, vc, bt = _paged(kk, v)
        sl = oracle.slopes(H, torch.float32)
        for lo in (0, 100, n - 1):
            got = ref.gqa_attention_biased(q[lo:], kc, vc, bt, torch.tensor([0, n - lo]), torch.tensor([n]), 0.4, window, 30.0, sl)
            assert torch.allclose(got.view(n - lo, H, vd), want[lo:], atol=1e-5)
        if 0 < dist < window and j >= 0 and dist < 20:      # it shows: leaving it out changes the result
            off = oracle.window_attention(q, kk, v, 0.4, 30.0, window, hide=lambda i, m: [j])
            assert float((off - want)[n - 1, 0].abs().max()) > 1e-2
    gate = torch.randn(n, H, generator=g)
    got = ref.gqa_attention_biased(q, kc, vc, bt, torch.tensor([0, n]), torch.tensor([n]), 0.4, window, 30.0, sl, gate, 0.3)
    assert torch.allclose(got.view(n, H, vd), 0.3 * want * oracle.sigmoid(gate)[:, :, None], atol=1e-5)


@pytest.mark.parametrize("m", [dict(heads=6, vdim=10, state=14, groups=3, conv=3, norm_groups=4), dict(heads=2, vdim=16, state=8, groups=1, conv=1, norm_groups=1),
                               dict(heads=4, vdim=8, state=24, groups=4, conv=6, norm_groups=2)])
def test_mamba2_statement(m):
    D, n, eps = 40, 23, 1e-3
    cfg = {"vocab": 8, "width": D, "streams": 1, "max_positions": 4, "norm": {"eps": eps}, "layers": [{"type": "mamba2", "mixer": m, "mlp": None}]}
    W = {k: v.float() for k, v in oracle.random_weights(cfg, 5).items()}
    h = torch.randn(n, D, generator=_g(1))
    p = "l0.mix."
    H, vd, N, G, K = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    C = H * vd + 2 * G * N
    a = h @ W[p + "in"].T
    proj, dt = a[:, : H * vd + C], a[:, H * vd + C:]
    win, st = torch.randn(3, K - 1, C), torch.randn(3, H, vd, N)              # stale: a fresh sequence ignores both
    outs = []
    for lo, hi in ((0, 9), (9, 10), (10, 12), (12, n)):
        outs.append(ref.mamba2_mix(proj[lo:hi], dt[lo:hi], W[p + "conv"], W[p + "conv.b"], W[p + "A_log"], W[p + "dt_bias"], W[p + "D"], W[p + "norm"], m["norm_groups"],
                                   win, st, torch.tensor([2]), torch.tensor([0, hi - lo]), torch.tensor([int(lo == 0)]), H, G, vd, N, eps))
    want = oracle.mamba2(h.double(), {k: v.double() for k, v in W.items()}, p, m, eps)
    assert torch.allclose(torch.cat(outs) @ W[p + "o"].T, want.float(), atol=2e-5)


@pytest.mark.parametrize("H,d,vd,decay", [(3, 10, 14, [0.5, 0.9, 0.999]), (2, 8, 24, [0.0, 1.0])])
def test_lightning_statement(H, d, vd, decay):
    D, n, eps = 32, 21, 1e-3
    W = {"r." + c: torch.randn(H * w, D, generator=_g(i)) * D ** -0.5 for i, (c, w) in enumerate((("q", d), ("k", d), ("v", vd), ("g", vd)))}
    W["r.norm"], W["r.o"] = 1 + 0.2 * torch.randn(H * vd, generator=_g(8)), torch.eye(H * vd)
    h = torch.randn(n, D, generator=_g(9))
    pr = {c: h @ W["r." + c].T for c in "qkvg"}
    st, outs = torch.randn(3, H, vd, d), []
    for lo, hi in ((0, 9), (9, 10), (10, 12), (12, n)):
        outs.append(ref.lightning_mix(*(pr[c][lo:hi] for c in "qkvg"), torch.tensor(decay), W["r.norm"], st, torch.tensor([1]), torch.tensor([0, hi - lo]),
                                      torch.tensor([int(lo == 0)]), H, d, vd, eps, 0.7))
    want = 0.7 * oracle.right_mixer(h.double(), {k: v.double() for k, v in W.items()}, "r.", {"heads": H, "dim": d, "vdim": vd, "decay": decay}, eps)
    assert torch.allclose(torch.cat(outs), want.float(), atol=2e-5)


# ---- the engine ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_single_tokens_agree_with_the_oracle(name, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=5.0)
    toks = tokens(150, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", "cpu", pages=4)
    for cuts in ([150], [2], [1], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64], [129, 1]):
        assert error(feed_all(llm, None, toks, cuts), want) < TOL, cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 4 and llm.engine.scheduler.num_fed() == 0


def test_a_single_key_shows_inside_its_window_and_not_outside(tmp_path):
    """Queries scaled until single keys stand out: hiding one key from the oracle changes the logits, and so does a window that is one token
    longer or shorter; the engine agrees with the oracle - in one prompt and token by token."""
    cfg, W, path = build("aligned", tmp_path, sharp=8.0)
    toks = tokens(140, cfg["vocab"], 4)
    want = oracle.forward(cfg, W, toks)
    for key in (0, 63, 64, 127):
        assert error(oracle.forward(cfg, W, toks, hide=lambda i, n: [key] if i > key + 1 else []), want) > 100 * TOL, key
    for off in (-1, 1):
        other = json.loads(json.dumps(cfg))
        for L in other["layers"]:
            if L["type"] == "parallel":
                L["mixer"]["left"]["mask"]["size"] += off
        assert error(oracle.forward(other, W, toks), want) > 20 * TOL, off
    llm = make_llm(path, "float32", "cpu", pages=4)
    assert error(feed_all(llm, None, toks, [140]), want) < TOL
    assert error(feed_all(llm, None, toks, [100, 1]), want) < TOL


def test_bfloat16_stays_near_the_oracle(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    toks = tokens(90, cfg["vocab"], 2)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "bfloat16", "cpu", pages=4)
    assert error(feed_all(llm, None, toks, [50, 1, 9]), want) < 0.08


def test_mixed_batches_with_pages_and_slots_used_again(tmp_path):
    cfg, W, path = build("odd", tmp_path, sharp=3.0)
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


def test_greedy_generation_through_the_scheduler(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (70, 2, 33, 1, 64)]
    want = [oracle.greedy(cfg, W, p, 5) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    for kw in (dict(), dict(max_num_batched_tokens=16), dict(max_num_batched_tokens=65)):       # chunked prompts, cut anywhere
        llm = make_llm(path, "float32", "cpu", pages=9, **kw)
        outs = {o["seq_id"]: o["token_ids"] for o in llm.generate(prompts, sp)}
        assert [outs[i + 1] for i in range(len(prompts))] == want, kw


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
    """Keys, values, states and convolution windows of every layer move with a sequence (prefill engine -> decode engine)."""
    from nanoengine_b200.parallel.kv_transfer import KVMigrator, LocalTransport, connect_inproc
    cfg, W, path = build("aligned", tmp_path)
    pre, dec = make_llm(path, "float32", "cpu", pages=9, mode="prefill", engine_id="p"), make_llm(path, "float32", "cpu", pages=9, mode="decode", engine_id="d")
    kv = dec.engine.executor.runner.cache
    assert [f["name"] for f in kv.page_families()] == [f"{n}_{i}" for i in range(3) for n in ("key", "value")]
    assert [f["name"] for f in kv.slot_families()] == ["delta_state_0", "delta_state_1", "delta_conv_1", "delta_state_2", "delta_state_3"]
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


def test_fed_steps_past_the_learned_positions_are_refused(tmp_path):
    cfg, W, path = build("parallel_only", tmp_path)
    llm = LLM(Config(model=path, dtype="float32", device="cpu", max_num_seqs=2, num_kvcache_blocks=8, enable_prefix_caching=False, status_log_interval_s=0))
    with pytest.raises(ValueError):
        llm.feed([(1, [1] * 301)])
    assert llm.feed([(2, [1] * 299)]) is None and llm.feed([(2, [1])], [[0]]).shape == (1, 64)
    with pytest.raises(ValueError):
        llm.feed([(2, [1])])


def test_random_weights_cover_the_checkpoint_and_loading_is_strict(tmp_path):
    llm = LLM(Config(model="tiny-filasun", device="cpu", dtype="float32", num_kvcache_blocks=8, max_model_len=256, max_num_seqs=4))
    outs = llm.generate([[1, 2, 3, 4]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(outs[0]["token_ids"]) == 4
    assert PRESETS["filasun-7b"]().num_hidden_layers == 24
    cfg, W, _ = build("odd", tmp_path)
    for change in (lambda w: w.pop("l1.mix.dt_bias"), lambda w: w.pop("l0.mix.left.v.b"), lambda w: w.update(extra=torch.zeros(2))):
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
    """The command line, with a pool larger than the model's positions: logits in files, pages and slots given back."""
    cfg, W, path = build("odd", tmp_path)
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(66, cfg["vocab"], 1), tokens(5, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:], "want": [3]}, {"id": "a", "tokens": a[64:65], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[65:], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [4]}], "end": ["b"]}]
    r = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "640",
                        "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    wa, wb = oracle.forward(cfg, W, a), oracle.forward(cfg, W, b)
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
    assert error(read(0), wa[[0, 63]]) < TOL and error(read(1), torch.stack([wb[4], wa[64]])) < TOL and error(read(3), wb[4:5]) < TOL
    assert not (out / "2.f32").exists()
