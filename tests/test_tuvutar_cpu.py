"""Tuvutar on CPU: the reader of its configuration, every operator's PyTorch statement against the plain oracle, and the engine -
scheduler, pages, state slots, portions, mixed batches, generation - in 32-bit against the oracle's logits."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import tuvutar_oracle as oracle
from tuvutar_models import CONFIGS, build, delta, error, feed_all, latent, make_llm, tokens, write_checkpoint
from nanoengine_b200 import Config, LLM, SamplingParams
from nanoengine_b200.models.config import PRESETS, ModelConfig
from nanoengine_b200.ops import reference as ref

TOL = 3e-5
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- configuration -------------------------------------------------------------------------------------------------
def test_config_reads_every_layer_and_survives_a_round_trip():
    mc = ModelConfig.from_dict(CONFIGS["odd"])
    assert (mc.vocab_size, mc.hidden_size, mc.num_hidden_layers, mc.rms_norm_eps) == (97, 76, 4, 1e-5)
    again = ModelConfig.from_dict(json.loads(json.dumps(mc.to_dict())))
    for c in (mc, again):
        assert [c.layer_type(i) for i in range(4)] == ["full_attention", "linear_attention", "linear_attention", "full_attention"]
        assert c.kv_source_layer(3) == 0 and c.is_mla and c.is_hybrid_gdn
        a, b = c.layer_config(0), c.layer_config(2)
        assert (a.num_attention_heads, a.qk_nope_head_dim, a.qk_rope_head_dim, a.v_head_dim, a.kv_lora_rank, a.intermediate_size) == (3, 12, 4, 20, 28, 50)
        assert a.attn_scale == 0.31 and a.glu_act == ("gelu_tanh",) and b.intermediate_size == 30
        assert (b.linear_num_value_heads, b.linear_num_key_heads, b.linear_key_head_dim, b.linear_value_head_dim, b.linear_conv_kernel_dim) == (4, 4, 36, 18, 2)
    assert not ModelConfig.from_dict(CONFIGS["latent_only"]).is_hybrid_gdn


@pytest.mark.parametrize("bad", [
    [latent(2, 8, 4, 8, 16, src=0)], [delta(2, 2, 8, 8, 4), latent(2, 8, 4, 8, 16, src=0)],
    [latent(2, 8, 4, 8, 16), latent(2, 8, 4, 8, 24, src=0)], [latent(2, 8, 4, 8, 16), latent(2, 8, 4, 8, 16, src=0, base=7.0)],
    [latent(2, 8, 4, 8, 16), latent(2, 8, 4, 8, 16, src=0), latent(2, 8, 4, 8, 16, src=1)], [delta(3, 2, 8, 8, 4)],
    [dict(delta(2, 2, 8, 8, 4), type="convolution")]])
def test_config_refuses_layers_that_do_not_fit_together(bad):
    with pytest.raises(ValueError):
        ModelConfig.from_dict({"architecture": "Tuvutar", "vocab": 32, "width": 32, "norm": {"eps": 1e-6}, "layers": bad})


def test_engine_config_follows_the_context_and_refuses_layouts():
    mc = ModelConfig.from_dict(CONFIGS["odd"])
    c = Config(model="x", model_config=mc, max_model_len=200000)
    assert c.model_config.max_position_embeddings >= 200000 and c.kvcache_block_size == 64
    with pytest.raises(ValueError):
        Config(model="x", model_config=ModelConfig.from_dict(CONFIGS["odd"]), attention_tp=2)


# ---- operators against the oracle ------------------------------------------------------------------------------------
def test_residual_norm_and_embed_norm():
    g = torch.Generator().manual_seed(0)
    x, y = torch.randn(5, 37, generator=g), torch.randn(5, 37, generator=g)
    wp, wn = torch.randn(37, generator=g) * 0.3, torch.randn(37, generator=g) * 0.3
    h, x2 = ref.residual_norm(y, x, wp, wn, 1e-2)
    want = x + oracle.offset_norm(y, wp, 1e-2)
    assert torch.allclose(x2, want, atol=1e-6) and torch.allclose(h, oracle.offset_norm(want, wn, 1e-2), atol=1e-5)
    h, x0 = ref.embed_norm(torch.tensor([3, 0]), x, wn, 1e-2)
    assert torch.equal(x0, x[[3, 0]]) and torch.allclose(h, oracle.offset_norm(x[[3, 0]], wn, 1e-2), atol=1e-5)


@pytest.mark.parametrize("rot", [{"base": 500.0, "dims": 16}, {"base": 20000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 256, "fast": 32.0, "slow": 1.0}},
                                 {"base": 50.0, "dims": 12, "scaling": {"factor": 2.5, "original": 4096, "fast": 8.0, "slow": 2.0}},
                                 {"base": 1e4, "dims": 4, "scaling": {"factor": 40.0, "original": 8, "fast": 32.0, "slow": 1.0}}])
def test_rotary_table(rot):
    from nanoengine_b200.models.config import _yarn_of
    table = ref.rope_cos_sin_cache(rot["dims"], 700, rot["base"], _yarn_of(rot.get("scaling")))
    x = torch.randn(4, 3, rot["dims"], dtype=torch.float64)
    pos = torch.tensor([0, 1, 77, 699])
    assert (ref.apply_rope(x, pos, table, True) - oracle.rotate(x, pos, rot)).abs().max() < 2e-4


def test_gelu_and_delta_pieces():
    z = torch.linspace(-6, 6, 101, dtype=torch.float64)
    assert torch.allclose(ref.glu_act(z, torch.ones_like(z), ("gelu_tanh",)), oracle.gelu_tanh(z), atol=1e-9)
    x = torch.linspace(-40, 40, 81, dtype=torch.float64)
    assert torch.allclose(torch.nn.functional.softplus(x), oracle.softplus(x), atol=1e-8)


@pytest.mark.parametrize("m", [dict(heads=6, kv_heads=2, dim=10, vdim=14, conv=3), dict(heads=2, kv_heads=2, dim=16, vdim=8, conv=4),
                               dict(heads=3, kv_heads=1, dim=8, vdim=24, conv=6)])
def test_gated_delta_statement(m):
    D, n, eps = 40, 23, 1e-3
    cfg = {"vocab": 8, "width": D, "norm": {"eps": eps}, "layers": [{"type": "delta", "mixer": m, "mlp": None}]}
    W = {k: v.float() for k, v in oracle.random_weights(cfg, 5).items()}
    h = torch.randn(n, D, generator=torch.Generator().manual_seed(1))
    p = "l0.mix."
    proj = torch.cat([h @ W[p + s].T for s in "qkvg"], -1)
    ab = torch.cat([h @ W[p + s].T for s in "ab"], -1)
    cw = torch.cat([W[p + s + ".conv"] for s in "qkv"], 0)
    H, Hk, dk, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    win, st = torch.randn(3, K - 1, cw.shape[0]), torch.randn(3, H, dv, dk)       # stale: a fresh sequence ignores both
    outs = []
    for lo, hi in ((0, 9), (9, 10), (10, 12), (12, n)):
        outs.append(ref.gated_delta(proj[lo:hi], ab[lo:hi], cw, W[p + "A_log"], W[p + "dt_bias"], W[p + "norm"], win, st, torch.tensor([2]),
                                    torch.tensor([0, hi - lo]), torch.tensor([int(lo == 0)]), Hk, H, dk, dv, eps))
    want = oracle.delta_mixer(h.double(), {k: v.double() for k, v in W.items()}, p, m, eps)
    assert torch.allclose(torch.cat(outs) @ W[p + "o"].T, want.float(), atol=1e-5)


# ---- the engine ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_single_tokens_agree_with_the_oracle(name, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=6.0)
    toks = tokens(150, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", "cpu", pages=4)
    for cuts in ([150], [2], [1], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64], [129, 1]):
        assert error(feed_all(llm, None, toks, cuts), want) < TOL, cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 4 and llm.engine.scheduler.num_fed() == 0


def test_a_single_far_key_shows_and_is_seen(tmp_path):
    """Queries scaled until single keys stand out: hiding any one old key from the oracle changes its logits visibly, at page borders
    too, and the engine agrees with the oracle that sees all of them - in one prompt and token by token."""
    cfg, W, path = build("aligned", tmp_path, sharp=12.0)
    toks = tokens(140, cfg["vocab"], 4)
    want = oracle.forward(cfg, W, toks)
    for key in (0, 1, 63, 64, 127):
        faulty = oracle.forward(cfg, W, toks, hide=lambda i, n, key=key: [key] if i > key + 1 else [])
        assert error(faulty, want) > 100 * TOL, key
    shifted = oracle.forward(cfg, W, toks, hide=lambda i, n: [i])        # a causal limit that is one token off
    assert error(shifted, want) > 100 * TOL
    llm = make_llm(path, "float32", "cpu", pages=4)
    assert error(feed_all(llm, None, toks, [140]), want) < TOL
    assert error(feed_all(llm, None, toks, [100, 1]), want) < TOL


def test_bfloat16_stays_near_the_oracle(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    toks = tokens(90, cfg["vocab"], 2)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "bfloat16", "cpu")
    assert error(feed_all(llm, None, toks, [50, 1, 9]), want) < 0.08


def test_mixed_batches_with_pages_and_slots_used_again(tmp_path):
    cfg, W, path = build("odd", tmp_path, sharp=4.0)
    reqs = {i: tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate([130, 70, 3, 1, 66, 65, 40, 129])}
    want = {i: oracle.forward(cfg, W, t) for i, t in reqs.items()}
    llm = make_llm(path, "float32", "cpu", pages=9, slots=4)
    at, live, todo, got, ids = {}, [], list(reqs), {i: [] for i in reqs}, {}
    rng = np.random.default_rng(0)
    step = 0
    while todo or live:
        while todo and len(live) < 4:
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
    assert llm.engine.scheduler.num_free_blocks(0) == 9 and llm.engine.scheduler.num_free_state_slots(0) == 4


def test_greedy_generation_through_the_scheduler(tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (70, 2, 33, 1, 64)]
    want = [oracle.greedy(cfg, W, p, 5) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    for kw in (dict(), dict(max_num_batched_tokens=16), dict(max_num_batched_tokens=65)):       # chunked prompts, cut anywhere
        llm = make_llm(path, "float32", "cpu", **kw)
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
def test_cache_plan_families_and_migration_between_engines(tmp_path, transport):
    """Rows of every latent layer and states of every delta layer move with a sequence (prefill engine -> decode engine)."""
    from nanoengine_b200.parallel.kv_transfer import KVMigrator, LocalTransport, connect_inproc
    cfg, W, path = build("aligned", tmp_path)
    pre, dec = make_llm(path, "float32", "cpu", mode="prefill", engine_id="p"), make_llm(path, "float32", "cpu", mode="decode", engine_id="d")
    kv = dec.engine.executor.runner.cache
    assert [f["name"] for f in kv.page_families()] == ["latent_0", "latent_1"]
    assert [f["name"] for f in kv.slot_families()] == ["delta_state_0", "delta_conv_0", "delta_state_1", "delta_conv_1"]
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


def test_fed_steps_are_checked_and_change_nothing_when_refused(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    llm = make_llm(path, "float32", "cpu", pages=2, slots=2)
    sch = llm.engine.scheduler
    with pytest.raises(ValueError):
        llm.feed([])
    with pytest.raises(ValueError):
        llm.feed([(1, [])])
    with pytest.raises(ValueError):
        llm.feed([(1, [2]), (1, [3])])
    with pytest.raises(RuntimeError):
        llm.feed([(1, [1] * 65), (2, [1] * 65)])                # more pages than there are
    with pytest.raises(RuntimeError):
        llm.feed([(1, [1]), (2, [1]), (3, [1])])                # more sequences than slots
    with pytest.raises(ValueError):
        llm.feed([(1, [1] * 129)])                              # past max_model_len
    assert sch.num_free_blocks(0) == 2 and sch.num_free_state_slots(0) == 2 and sch.num_fed() == 0
    toks = tokens(70, cfg["vocab"], 6)
    assert error(feed_all(llm, None, toks, [70]), oracle.forward(cfg, W, toks)) < TOL
    assert llm.feed([(5, toks[:3])]) is None and llm.end_feed([5, 6]) == 1


def test_random_weights_cover_the_checkpoint_and_loading_is_strict(tmp_path):
    for preset in ("tiny-tuvutar",):
        llm = LLM(Config(model=preset, device="cpu", dtype="float32", num_kvcache_blocks=8, max_model_len=256, max_num_seqs=4))
        outs = llm.generate([[1, 2, 3, 4]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
        assert len(outs[0]["token_ids"]) == 4
    assert PRESETS["tuvutar-7b"]().num_hidden_layers == 32
    cfg, W, _ = build("odd", tmp_path)
    for change in (lambda w: w.pop("l1.mix.dt_bias"), lambda w: w.update(extra=torch.zeros(2))):
        w = dict(W)
        change(w)
        with pytest.raises(ValueError):
            make_llm(write_checkpoint(os.path.join(str(tmp_path), "bad"), cfg, w), "float32", "cpu")


def test_weights_can_be_replaced_in_place(tmp_path):
    cfg, W, path = build("odd", tmp_path)
    W2 = oracle.random_weights(cfg, 77)
    llm = make_llm(path, "float32", "cpu")
    llm.update_weights(list(W2.items()))
    toks = tokens(20, cfg["vocab"], 3)
    assert error(feed_all(llm, None, toks, [20]), oracle.forward(cfg, W2, toks)) < TOL


def test_replay_program(tmp_path):
    """The command line: steps on standard input, logits in files, requests that end give their pages and slots back."""
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
