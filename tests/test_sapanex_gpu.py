"""Sapanex on the GPU: every kernel against its 32-bit PyTorch statement, and the engine - prompts, portions, mixed batches, decode graphs,
generation - against the plain oracle, in true 32-bit and in bf16."""
import pytest
import torch

import sapanex_oracle as oracle
from sapanex_models import CONFIGS, YARN, build
from tuvutar_models import error, feed_all, make_llm, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.1}
ROUGH = {"delta_only": 0.15}        # how far bf16 rounding alone takes a model, where that is more than the rest


def _k():
    from nanoengine_b200.ops import sm100
    return sm100


def _ref():
    from nanoengine_b200.ops import reference
    return reference


def rel(a, b):
    return float((a.float().cpu() - b.float().cpu()).abs().max() / b.float().abs().max().clamp_min(1e-6))


def _cu(lens):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)


# ---- kernels -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K,at", [(1, 8, 64, 0), (3, 96, 72, 50), (70, 136, 128, 128), (129, 64, 200, 33), (128, 520, 4096, 515), (300, 4104, 512, 4000), (5, 97, 76, 90),
                                      (64, 20544, 256, 20480)])
@pytest.mark.parametrize("act", ["relu2", "tanh"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_activation_in_the_epilogue(M, N, K, at, act, dtype):
    k = _k()
    g = torch.Generator(device=DEV).manual_seed(M)
    x, w = torch.randn(M, K, generator=g, device=DEV).to(dtype), (torch.randn(N, K, generator=g, device=DEV) * K ** -0.5).to(dtype)
    z = x.double() @ w.double().T
    want = torch.cat([z[:, :at], z[:, at:].tanh() if act == "tanh" else z[:, at:].clamp_min(0).square()], -1)
    got = k.linear(x, w, act=act, act_from=at)
    assert rel(got, want) < (5e-6 if dtype == torch.float32 else 4.1e-3) and rel(got[:, at:], want[:, at:]) < (5e-6 if dtype == torch.float32 else 4.1e-3)
    assert rel(k.linear(x, w, out_fp32=True, act=act, act_from=at), want) < (5e-6 if dtype == torch.float32 else 1e-5)
    assert torch.equal(k.linear(x, w, act=act, act_from=N), k.linear(x, w))


@pytest.mark.parametrize("T,W", [(1, 76), (5, 128), (33, 320), (4, 4096), (2, 20000), (3, 51)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_behind_the_sum(T, W, dtype):
    k, r = _k(), _ref()
    g = torch.Generator(device=DEV).manual_seed(T + W)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    y, x, w, wl = (3 * rnd(T, W + 4)).to(dtype)[:, :W], rnd(T, W), (1 + 0.3 * rnd(W)).to(dtype), (1 + 0.3 * rnd(W)).to(dtype)
    tol = 5e-6 if dtype == torch.float32 else 5e-3
    for last in (None, wl):
        hw, xw = r.postnorm(y.float(), x.clone(), 2.5, w, 1e-3, last)
        h, x2 = k.postnorm(y, x.clone(), 2.5, w, 1e-3, last)
        assert h.dtype == dtype and rel(x2, xw) < 2e-6 and rel(h, hw) < tol
    table, ids = rnd(11, W).to(dtype), torch.randint(0, 11, (T,), generator=g, device=DEV)
    h, x0 = k.embed_scaled(ids, table, 6.5)
    assert torch.equal(x0, 6.5 * table[ids].float()) and torch.equal(h, x0.to(dtype))


@pytest.mark.parametrize("T", [1, 3])
def test_products_of_rows_that_start_anywhere(T):
    """The second factor of the decay's projection reads a slice of the merged projection, wherever that lies."""
    k = _k()
    y, w = torch.randn(T, 80, device=DEV).to(torch.bfloat16), torch.randn(16, 8, device=DEV).to(torch.bfloat16)
    for at in (60, 61, 64):
        assert rel(k.linear_fp32(y[:, at: at + 8], w), y[:, at: at + 8].double() @ w.double().T) < 1e-5


def _paged(q_lens, ctx, G, D, Dv, pool, dtype, g, page=64):
    pages = [(c + page - 1) // page for c in ctx]
    perm = torch.randperm(sum(pages) + 3, generator=g, device=DEV)
    bt = torch.zeros(len(ctx), max(pages), dtype=torch.int32, device=DEV)
    at = 0
    for i, n in enumerate(pages):
        bt[i, :n] = perm[at: at + n].int()
        at += n
    rnd = lambda r, w: torch.randn(sum(pages) + 3, r, G, w, generator=g, device=DEV).to(dtype)
    rows = _ref().pooled_rows_per_page(pool, page)
    return rnd(page, D), rnd(page, Dv), rnd(rows, D), rnd(rows, Dv), bt, _cu(q_lens), torch.tensor(ctx, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 56, 40), (6, 2, 80, 24), (8, 8, 128, 128), (32, 4, 128, 64), (5, 1, 64, 256), (24, 2, 256, 200), (128, 1, 72, 8), (16, 16, 64, 72),
                                      (3, 1, 12, 20), (10, 2, 17, 6)])
@pytest.mark.parametrize("window,pool,turned", [(70, 5, True), (64, 64, True), (1, 1, False), (33, 16, True), (200, 130, False), (5, 3, True)])
@pytest.mark.parametrize("q_lens,ctx", [([1, 1, 1], [1, 64, 700]), ([5, 130, 1, 33], [5, 200, 129, 1095])])
def test_window_and_pooled_blocks(H, G, D, Dv, window, pool, turned, q_lens, ctx):
    """Shuffled pages against the 32-bit statement, on the tensor cores where the sizes allow it and on the generic kernel; for the last query of
    each sequence the last key of its window, the one before it, the last block it sees and the next one stand out."""
    from nanoengine_b200.ops import sm100_attn
    place = _ref().pooled_row_place
    for dtype in (torch.bfloat16, torch.float32):
        g = torch.Generator(device=DEV).manual_seed(H + D)
        T = sum(q_lens)
        kc, vc, kp, vp, bt, cu, cl = _paged(q_lens, ctx, G, D, Dv, pool, dtype, g)
        q = torch.randn(T, H * D + (8 - H * D % 8) % 8, generator=g, device=DEV).to(dtype)[:, : H * D].unflatten(-1, (H, D))
        row, h = 0, H // 2
        for i, n in enumerate(q_lens):
            row += n
            for j in (ctx[i] - window, ctx[i] - 1 - window):
                if 0 <= j < ctx[i] - 1:
                    kc[bt[i, j // 64], j % 64, h // (H // G)] = q[row - 1, h] * 0.5
            seen = max(0, (ctx[i] - window) // pool)
            for b in (seen - 1, seen):
                if 0 <= b and (b + 1) * pool <= ctx[i]:
                    pg, r = place(b, pool, 64)
                    kp[bt[i, pg], r, h // (H // G)] = q[row - 1, h] * 0.5
        table = torch.randn(max(ctx), Dv, generator=g, device=DEV) if turned else None
        f = lambda t: t.float()
        want = _ref().gqa_attention_biased(f(q), f(kc), f(vc), bt, cu, cl, 1.3 * D ** -0.5, window, pooled=(f(kp), f(vp)), pool=pool, turn_back=table)
        on_tc = dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0
        for splits in (None, 1, 3) if on_tc else (None,):
            y = torch.zeros(T, H * Dv + 8, device=DEV, dtype=dtype)
            before = sm100_attn.BIASED_TC_CALLS[0]
            sm100_attn.gqa_attention_biased(q, kc, vc, bt, cu, cl, 1.3 * D ** -0.5, window, out=y[:, : H * Dv], max_q_len=max(q_lens), pooled=(kp, vp), pool=pool,
                                            turn_back=table, splits=splits)
            assert sm100_attn.BIASED_TC_CALLS[0] == before + int(on_tc)
            assert rel(y[:, : H * Dv], want) < (1e-2 if dtype == torch.bfloat16 else 5e-6), (dtype, splits)
            assert float(y[:, H * Dv:].abs().max()) == 0.0
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("H,G,D,Dv,rot,pool", [(4, 2, 48, 72, 24, 11), (6, 2, 12, 10, 6, 7), (5, 1, 9, 14, 8, 23), (8, 8, 40, 56, 24, 3), (32, 8, 128, 128, 64, 16),
                                               (2, 2, 16, 40, 16, 70), (1, 1, 8, 8, 2, 1)])
@pytest.mark.parametrize("starts,lens,page", [([0, 63, 200], [1, 1, 1], 64), ([0, 100, 37, 69], [130, 1, 2, 90], 64), ([11, 5], [60, 1], 16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_front_end(H, G, D, Dv, rot, pool, starts, lens, page, dtype):
    k, r = _k(), _ref()
    g = torch.Generator(device=DEV).manual_seed(H * D)
    T, ctx = sum(lens), [s + n for s, n in zip(starts, lens)]
    kc, vc, kp, vp, bt, cu, _ = _paged(lens, ctx, G, D, Dv, pool, dtype, g, page)
    pos = torch.cat([torch.arange(s, s + n, device=DEV) for s, n in zip(starts, lens)])
    seq = torch.repeat_interleave(torch.arange(len(lens), device=DEV), torch.tensor(lens, device=DEV))
    slots = bt[seq, pos // page].long() * page + pos % page
    if T > len(lens):
        slots[1] = -1                                          # a padded token writes nothing
    from nanoengine_b200.models.config import _yarn_of
    kt = r.rope_cos_sin_cache(rot, max(ctx), 1000.0, _yarn_of(YARN), exact=True).to(DEV)
    vt = r.rope_cos_sin_cache(Dv, max(ctx), 1000.0, exact=True).to(DEV)
    qkv = torch.randn(T, H * D + G * (D + Dv) + 3, generator=g, device=DEV).to(dtype)[:, : H * D + G * (D + Dv)]
    qn, kn = ((1 + 0.3 * torch.randn(n, generator=g, device=DEV)).to(dtype) for n in (H * D, G * D))
    want = [t.clone() for t in (kc, vc, kp, vp)]
    q_want = r.pooled_attention_prepare(qkv.clone(), H, G, D, Dv, qn, kn, 1e-2, pos, kt, vt, *want, pool, slots, bt, cu, max(lens))
    q = k.pooled_attention_prepare(qkv.clone(), H, G, D, Dv, qn, kn, 1e-2, pos, kt, vt, kc, vc, kp, vp, pool, slots, bt, cu, max(lens))
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    assert rel(q, q_want) < tol
    for a, b in zip((kc, vc, kp, vp), want):
        assert rel(a, b) < tol
    assert k.kernel_status()[0] == 0


LENS = [([1, 1, 1], [0, 0, 1]), ([37, 1, 2, 9], [1, 0, 0, 1]), ([2, 1], [0, 0]), ([8, 16, 17], [0, 1, 0]), ([200, 1, 129], [0, 0, 1])]


def _delta_case(H, Dk, Dv, lens, fresh, dtype, seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    T, B = sum(lens), len(lens)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    return dict(proj=rnd(T, H * (3 * Dk + 2 * Dv) + 8).to(dtype), decay=rnd(T, H * Dk + (4 - H * Dk % 4) % 4), w0=1.5 * rnd(H * Dk) - 2, a_bias=rnd(H * Dk),
                norm_w=(1 + 0.2 * rnd(H * Dv)).to(dtype), state=0.3 * rnd(B + 2, H, Dv, Dk), slots=torch.randperm(B + 2, generator=g, device=DEV)[:B].int(),
                cu_seqlens=_cu(lens), fresh=torch.tensor(fresh, dtype=torch.int32, device=DEV), H=H, Dk=Dk, Dv=Dv, eps=1e-4, max_q_len=max(lens))


def _copy(c):
    return {n: (v.clone() if isinstance(v, torch.Tensor) else v) for n, v in c.items()}


def _delta64(c):
    """The statement in 64-bit: a head whose output nearly vanishes is scaled up by its own norm, which 32-bit statements differ by."""
    H, Dk, Dv, cu, state = c["H"], c["Dk"], c["Dv"], c["cu_seqlens"].tolist(), c["state"].double()
    T, nk, nv = c["proj"].shape[0], H * Dk, H * Dv
    r, k, a, v, gate = c["proj"].double()[:, : 3 * nk + 2 * nv].split([nk, nk, nk, nv, nv], -1)
    w = torch.exp(-torch.exp(torch.tensor(-0.5, dtype=torch.float64)) * torch.sigmoid(c["decay"].double()[:, :nk] + c["w0"])).view(T, H, Dk)
    a = torch.sigmoid(a + c["a_bias"]).view(T, H, Dk)
    r, k, v, o = r.reshape(T, H, Dk), k.reshape(T, H, Dk), v.reshape(T, H, Dv), torch.empty(T, H, Dv, dtype=torch.float64, device=DEV)
    for i, slot in enumerate(c["slots"].tolist()):
        s, e = cu[i], cu[i + 1]
        S = torch.zeros_like(state[slot]) if int(c["fresh"][i]) else state[slot].clone()
        o[s:e], state[slot] = _ref().general_delta_scan(r[s:e], k[s:e], v[s:e], w[s:e], a[s:e], S)
    o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + c["eps"])
    return o.reshape(T, nv) * c["norm_w"] * torch.sigmoid(gate), state


@pytest.mark.parametrize("H,Dk,Dv", [(3, 10, 10), (4, 64, 64), (2, 128, 128), (4, 32, 32), (8, 16, 64), (1, 72, 16), (2, 17, 5), (2, 200, 96), (1, 144, 144), (3, 96, 40), (1, 300, 33),
                                     (40, 128, 128)])
@pytest.mark.parametrize("lens,fresh", LENS)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_general_delta(H, Dk, Dv, lens, fresh, dtype):
    c = _delta_case(H, Dk, Dv, lens, fresh, dtype)
    want_out, want_state = _delta64(c)
    out = _k().general_delta(**c)
    assert rel(c["state"], want_state) < 5e-6 and rel(out, want_out) < (5e-5 if dtype == torch.float32 else 6e-3)
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("H,D", [(4, 64), (48, 128), (2, 30), (1, 160)])
def test_the_recurrence_does_not_depend_on_the_cut(H, D):
    n = 300
    c = _delta_case(H, D, D, [n], [1], torch.bfloat16)
    whole = _copy(c)
    out = _k().general_delta(**whole)
    at, got = 0, []
    for m in (1, 2, 33, 1, 1, 128, 65, 2, 67):
        part = dict(c, cu_seqlens=_cu([m]), fresh=torch.tensor([int(at == 0)], dtype=torch.int32, device=DEV), max_q_len=m, **{r: c[r][at: at + m] for r in ("proj", "decay")})
        got.append(_k().general_delta(**part))
        at += m
    assert at == n and rel(c["state"], whole["state"]) < 1e-5 and rel(torch.cat(got), out) < 5e-3


# ---- the engine ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_engine_agrees_with_the_oracle(name, dtype, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=2.0 if dtype == "float32" else 1.5)
    toks = tokens(200, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, dtype, DEV, pages=4)
    for cuts in ([200], [130, 1], [2], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64]):
        assert error(feed_all(llm, None, toks, cuts), want) < (ROUGH.get(name, TOL[dtype]) if dtype == "bfloat16" else TOL[dtype]), cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 4
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_requests_alone(dtype, tmp_path):
    cfg, W, path = build("aligned", tmp_path)
    reqs = {i: tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate([130, 70, 3, 66])}
    want = {i: oracle.forward(cfg, W, t) for i, t in reqs.items()}
    llm = make_llm(path, dtype, DEV, pages=9)
    at, got = {i: 0 for i in reqs}, {i: [] for i in reqs}
    sizes = {0: [64, 1, 1, 63, 1], 1: [1, 1, 33, 1, 34], 2: [1, 1, 1], 3: [2, 1, 1, 1, 1, 60]}
    for step in range(6):
        entries, wants, who = [], [], []
        for i in reqs:
            if step < len(sizes[i]):
                n = sizes[i][step]
                entries.append((i + 1, reqs[i][at[i]: at[i] + n])); wants.append(list(range(n))); who.append((i, n))
                at[i] += n
        out, row = torch.from_numpy(llm.feed(entries, wants)), 0
        for i, n in who:
            got[i].append(out[row: row + n]); row += n
    for i in reqs:
        assert error(torch.cat(got[i]), want[i]) < TOL[dtype], i
    llm.end_feed([1, 2, 3, 4])


def test_pages_and_slots_used_again(tmp_path):
    """Requests one after the other through a pool of three pages and one slot: what an earlier one left in pages, pooled rows and states does not
    show."""
    cfg, W, path = build("odd", tmp_path)
    llm = make_llm(path, "float32", DEV, pages=3, slots=1)
    for seed, n in enumerate((190, 30, 129, 64, 65, 2)):
        toks = tokens(n, cfg["vocab"], seed)
        assert error(feed_all(llm, None, toks, [n // 2 + 1, 1, 2], seq_id=seed + 1), oracle.forward(cfg, W, toks)) < TOL["float32"], n


def test_generation_in_32_bit_equals_the_oracle_and_graphs_equal_eager(tmp_path):
    from nanoengine_b200 import SamplingParams
    cfg, W, path = build("aligned", tmp_path)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (70, 2, 33, 1, 64)]
    want = [oracle.greedy(cfg, W, p, 6) for p in prompts]
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    for kw in (dict(), dict(enforce_eager=True), dict(max_num_batched_tokens=16)):
        llm = make_llm(path, "float32", DEV, pages=9, **kw)
        outs = {o["seq_id"]: o["token_ids"] for o in llm.generate(prompts, sp)}
        assert [outs[i + 1] for i in range(len(prompts))] == want, kw
    llm = make_llm(path, "bfloat16", DEV, pages=9)
    for p in prompts[:3]:
        llm.add_request(p, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for _ in range(6):
        llm.step()
    runner = llm.engine.executor.runner
    assert runner.graphs is not None and runner.graphs.graphs and runner.graph_step_equals_eager()


@pytest.mark.parametrize("name", ["fine", "attention_only"])
def test_long_decoding(name, tmp_path):
    """Several hundred single tokens through the decode graph: every token completes or does not complete a block, keys leave the window, blocks come
    into sight."""
    cfg, W, path = build(name, tmp_path, sharp=2.0)
    toks = tokens(500, cfg["vocab"], 8)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", DEV, pages=8)
    assert error(feed_all(llm, None, toks, [20, 1]), want) < TOL["float32"]


def test_pool_sized_from_the_free_memory(tmp_path):
    import gc
    gc.collect()                                # what earlier tests hold counts as used
    torch.cuda.empty_cache()
    from nanoengine_b200 import LLM, Config, SamplingParams
    cfg, W, path = build("odd", tmp_path)
    llm = LLM(Config(model=path, dtype="bfloat16", device=DEV, max_num_seqs=4, max_num_batched_tokens=1000, max_model_len=4096, gpu_memory_utilization=0.15,
                     executor_backend="inproc", enable_prefix_caching=False, status_log_interval_s=0))
    assert llm.engine.scheduler.num_free_blocks(0) > 100
    out = llm.generate([tokens(70, cfg["vocab"], 1)], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(out[0]["token_ids"]) == 4 and _k().kernel_status()[0] == 0
