"""Gipozen on the GPU: every kernel against its 32-bit PyTorch statement, and the engine - prompts, portions, mixed batches, decode graphs,
generation - against the plain oracle, in true 32-bit and in bf16."""
import pytest
import torch

import gipozen_oracle as oracle
from gipozen_models import CONFIGS, build
from tuvutar_models import error, feed_all, make_llm, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.1}
BOTH = [torch.float32, torch.bfloat16]


def _k():
    from nanoengine_b200.ops import sm100
    return sm100


def _ref():
    from nanoengine_b200.ops import reference
    return reference


def rel(a, b):
    return float((a.double().cpu() - b.double().cpu()).abs().max() / b.double().abs().max().clamp_min(1e-6))


def _cu(lens):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)


def _rnd(seed):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return g, lambda *s: torch.randn(*s, generator=g, device=DEV)


# ---- kernels -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,W,layers", [(1, 76, 1), (5, 128, 4), (33, 320, 7), (4, 4096, 25), (2, 20000, 3), (3, 51, 60)])
@pytest.mark.parametrize("dtype", BOTH)
def test_depth_average(T, W, layers, dtype):
    k, r = _k(), _ref()
    g, rnd = _rnd(T + W)
    tol = 5e-6 if dtype == torch.float32 else 5e-3
    table, ids, n = rnd(11, W).to(dtype), torch.randint(0, 11, (T,), generator=g, device=DEV), torch.tensor([0.8], device=DEV)
    h, x, bank = k.depth_embed(ids, table, n, 1e-3, layers + 1)
    hw, xw, _ = r.depth_embed(ids, table.float(), n, 1e-3, layers + 1)
    assert torch.equal(x, xw) and torch.equal(bank[0], xw) and h.dtype == dtype and rel(h, hw) < tol
    bank.copy_(rnd(layers + 1, T, W))
    y, w = rnd(T, W + 4).to(dtype)[:, :W], rnd(layers + 1)
    hw, mid = r.depth_mix(y.float(), x.clone(), n, 1e-3)
    h, x = k.depth_mix(y, x, n, 1e-3)
    assert rel(x, mid) < 2e-6 and rel(h, hw) < tol
    want_bank = bank.clone()
    hw, xw = r.depth_mix(y.float(), x.clone(), n, 1e-3, want_bank, layers, w)
    before, x_before = bank.clone(), x.clone()
    h, x2 = k.depth_mix(y, x, n, 1e-3, bank, layers, w, last=True)
    assert rel(h, hw) < tol and torch.equal(bank, before) and torch.equal(x, x_before)
    h, x = k.depth_mix(y, x, n, 1e-3, bank, layers, w)
    assert rel(h, hw) < tol and rel(x, xw) < 5e-6 and rel(bank, want_bank) < 2e-6
    assert k.kernel_status()[0] == 0


@pytest.mark.parametrize("T,F", [(1, 50), (7, 128), (33, 1536), (3, 24576), (5, 101)])
@pytest.mark.parametrize("dtype", BOTH)
def test_normed_powers(T, F, dtype):
    _, rnd = _rnd(F)
    z, coef = (2 * rnd(T, F + 4)).to(dtype)[:, :F], torch.tensor([1.1, -0.4, 0.3, 0.2], device=DEV)
    assert rel(_k().poly_norm(z, coef, 1e-4), _ref().poly_norm(z.double(), coef.double(), 1e-4)) < (5e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("qw,G,kd,vd", [(96, 2, 48, 24), (33, 3, 5, 7), (2048, 4, 128, 128), (64, 0, 0, 0)])
@pytest.mark.parametrize("starts,lens", [([0, 63, 200], [1, 1, 1]), ([0, 100, 37, 69, 0], [130, 1, 2, 90, 3]), ([11], [17])])
@pytest.mark.parametrize("dtype", BOTH)
def test_short_convolution(taps, qw, G, kd, vd, starts, lens, dtype):
    k, r = _k(), _ref()
    g, rnd = _rnd(taps * qw)
    T, C, B, page = sum(lens), qw + G * (kd + vd), len(lens), 64
    kc, vc = (rnd(9, page, G, d).to(dtype) if G else None for d in (kd, vd))
    rows = torch.randperm(9 * page, generator=g, device=DEV)[:T]
    if T > B:
        rows[1] = -1                                          # a padded token stores no rows
    u, w, win = rnd(T, C + 16).to(dtype), rnd(taps, C).to(dtype), rnd(B + 2, taps - 1, C).to(dtype)
    slots, fresh = torch.randperm(B + 2, generator=g, device=DEV)[:B].int(), torch.tensor([int(s == 0) for s in starts], dtype=torch.int32, device=DEV)
    want = [None if t is None else t.clone() for t in (kc, vc, win)]
    args = (slots, _cu(lens), fresh, max(lens))
    q_want = r.conv_rows(u, w, qw, *want[:2], rows, want[2], *args)
    q = k.conv_rows(u, w, qw, kc, vc, rows, win, *args)
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    assert rel(q, q_want) < tol and torch.equal(win, want[2])
    if G:
        assert rel(kc, want[0]) < tol and rel(vc, want[1]) < tol
    assert k.kernel_status()[0] == 0


@pytest.mark.parametrize("dtype", BOTH)
def test_convolution_does_not_depend_on_the_cut(dtype):
    _, rnd = _rnd(1)
    n, C = 200, 136
    u, w = rnd(n, C).to(dtype), rnd(4, C).to(dtype)
    run = lambda part, win, fresh: _k().conv_rows(part, w, C, None, None, torch.zeros(part.shape[0], dtype=torch.long, device=DEV), win, torch.zeros(1, dtype=torch.int32, device=DEV),
                                                  _cu([part.shape[0]]), torch.tensor([fresh], dtype=torch.int32, device=DEV), part.shape[0])
    win = rnd(1, 3, C).to(dtype)
    whole = run(u, win.clone(), 1)
    at, got = 0, []
    for m in (1, 2, 33, 1, 1, 1, 100, 2, 59):
        got.append(run(u[at: at + m], win, int(at == 0)))
        at += m
    assert at == n and torch.equal(torch.cat(got), whole)


def _paged(q_lens, ctx, G, kd, vd, dtype, g, page=64):
    pages = [(c + page - 1) // page for c in ctx]
    perm = torch.randperm(sum(pages) + 3, generator=g, device=DEV)
    bt = torch.zeros(len(ctx), max(pages), dtype=torch.int32, device=DEV)
    at = 0
    for i, n in enumerate(pages):
        bt[i, :n] = perm[at: at + n].int()
        at += n
    rnd = lambda w: torch.randn(sum(pages) + 3, page, G, w, generator=g, device=DEV).to(dtype)
    return rnd(kd), rnd(vd), bt, _cu(q_lens), torch.tensor(ctx, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 56, 40), (6, 2, 80, 24), (8, 8, 128, 128), (32, 4, 64, 128), (5, 1, 64, 256), (16, 2, 128, 256), (64, 1, 72, 8), (16, 16, 64, 72),
                                      (3, 1, 12, 20), (10, 2, 17, 6), (2, 1, 8, 8), (3, 3, 120, 200)])
@pytest.mark.parametrize("window,keep", [(70, 5), (64, 64), (1, 1), (33, 130), (200, 0), (5, 3), (0, 0)])
@pytest.mark.parametrize("q_lens,ctx", [([1, 1, 1], [1, 64, 700]), ([5, 130, 1, 33], [5, 200, 129, 1095])])
def test_differential_attention(H, G, D, Dv, window, keep, q_lens, ctx):
    """Shuffled pages against the 32-bit statement, on the tensor cores where the sizes allow it and on the generic kernel; for the last query of
    each sequence the last key of its window, the one before it, the last kept token and the next one stand out in one map or the other."""
    from nanoengine_b200.ops import sm100_attn
    for dtype in (torch.bfloat16, torch.float32):
        g, rnd = _rnd(H + D)
        T = sum(q_lens)
        kc, vc, bt, cu, cl = _paged(q_lens, ctx, G, 2 * D, Dv, dtype, g)
        q = rnd(T, H * 2 * D + (8 - H * 2 * D % 8) % 8).to(dtype)[:, : H * 2 * D].unflatten(-1, (H, 2, D))
        row, h = 0, H // 2
        for i, n in enumerate(q_lens):
            row += n
            for m, j in ((0, ctx[i] - window), (1, ctx[i] - 1 - window), (1, keep - 1), (0, keep)):
                if 0 <= j < ctx[i] - 1:
                    kc[bt[i, j // 64], j % 64, h // (H // G), m * D: (m + 1) * D] = q[row - 1, h, m] * 0.5
        gate, mixing = rnd(T, H * Dv + 8).to(dtype)[:, : H * Dv], torch.tensor([0.37], device=DEV)
        f = lambda t: t.float()
        want = _ref().differential_attention(f(q), f(kc), f(vc), bt, cu, cl, 1.3 * D ** -0.5, window, keep, mixing, 0.6, 1e-3, f(gate))
        on_tc = dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0
        for splits in (None, 1, 3) if on_tc else (None,):
            before = sm100_attn.DIFF_TC_CALLS[0]
            y = sm100_attn.differential_attention(q, kc, vc, bt, cu, cl, 1.3 * D ** -0.5, window, keep, mixing, 0.6, 1e-3, gate, max(q_lens), splits=splits)
            assert sm100_attn.DIFF_TC_CALLS[0] == before + int(on_tc)
            assert rel(y, want) < (2e-2 if dtype == torch.bfloat16 else 1e-5), (dtype, splits)
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("T,E,identity,top,gate", [(1, 5, 2, 3, 1), (37, 64, 8, 6, 1), (300, 200, 0, 8, 0), (9, 3, 3, 6, 0)])
def test_routing_by_corrected_scores(T, E, identity, top, gate):
    _, rnd = _rnd(E)
    logits, corr = 2 * rnd(T, E + identity + gate), 0.2 * rnd(E + identity)
    for planes in (logits, torch.stack([0.25 * logits, 0.75 * logits])):
        kw = dict(norm_topk_prob=False, scoring="softmax", gate_cols=gate, split_gate=True)
        idx, w, gt = _k().moe_route(planes, corr, top, **kw)
        iw, ww, gw = _ref().moe_route(planes, corr, top, **kw)
        assert torch.equal(idx.sort(-1).values, iw.sort(-1).values) and rel(w.sum(-1), ww.sum(-1)) < 1e-6
        assert torch.allclose(w.gather(1, idx.argsort(-1)), ww.gather(1, iw.argsort(-1)), atol=1e-6)
        assert (gt is None and gw is None) if not gate else torch.allclose(gt, gw, atol=1e-6)


@pytest.mark.parametrize("T,D,E,identity,top,F,shared", [(1, 128, 6, 2, 3, 64, 96), (70, 256, 12, 4, 5, 128, 0), (33, 192, 5, 0, 1, 72, 40), (130, 76, 7, 3, 8, 30, 50),
                                                         (300, 512, 40, 8, 6, 256, 256), (5, 320, 3, 1, 2, 200, 104)])
@pytest.mark.parametrize("dtype", BOTH)
def test_mixture(T, D, E, identity, top, F, shared, dtype):
    """The whole block on the GPU against the same block in 64-bit on the CPU."""
    from nanoengine_b200.models.layers import GatedSharedMoE
    g = torch.Generator().manual_seed(D)
    act, sact = ("clamp_linear", 0.9, 1.702), ("clamp_linear", 0.5, 1.702)
    M = GatedSharedMoE(D, E, identity, top, F, act, shared, sact if shared else None, dtype, DEV)
    R = GatedSharedMoE(D, E, identity, top, F, act, shared, sact if shared else None, torch.float64, "cpu")
    for (n, p), q in zip(M.named_parameters(), R.parameters()):
        t = torch.randn(q.shape, generator=g, dtype=torch.float64) * (0.05 if n == "correction" else q.shape[-1] ** -0.5)
        p.copy_(t)
        q.copy_(p.double().cpu())
    x = torch.randn(T, D, generator=g).to(dtype)
    idx, _, _ = _ref().moe_route(_ref().router_logits(x, R.router_weight), R.correction, top, norm_topk_prob=False, scoring="softmax", gate_cols=int(shared > 0), split_gate=True)
    assert rel(M(x.to(DEV)), R(x.double())) < (1e-5 if dtype == torch.float32 else 1.5e-2)
    if identity and T > 30:
        assert int((idx >= E).sum()) > 0
    assert _k().kernel_status()[0] == 0


# ---- the engine ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_engine_agrees_with_the_oracle(name, dtype, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=2.0 if dtype == "float32" else 1.0)
    toks = tokens(200, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, dtype, DEV, pages=4)
    for cuts in ([200], [130, 1], [2], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64]):
        assert error(feed_all(llm, None, toks, cuts), want) < TOL[dtype], cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 4
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_requests_alone(dtype, tmp_path):
    cfg, W, path = build("aligned", tmp_path, sharp=1.0)
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
    """Requests one after the other through a pool of three pages and one slot: what an earlier one left in pages and windows does not show."""
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


@pytest.mark.parametrize("name", ["fine", "stateless"])
def test_long_decoding(name, tmp_path):
    """Several hundred single tokens through the decode graph: keys leave the windows, kept tokens stay."""
    cfg, W, path = build(name, tmp_path, sharp=2.0)
    toks = tokens(400, cfg["vocab"], 8)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", DEV, pages=7)
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
