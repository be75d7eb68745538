"""Filasun on the GPU: every kernel against its 32-bit PyTorch statement, and the engine - prompts, portions, mixed batches, decode graphs,
generation - against the plain oracle, in true 32-bit and in bf16."""
import pytest
import torch

import filasun_oracle as oracle
from filasun_models import CONFIGS, build
from tuvutar_models import error, feed_all, make_llm, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.08}
ROUGH = {"mamba_only": 0.2}        # how far bf16 rounding alone takes a model, where that is more than the rest


def _k():
    from nanoengine_b200.ops import sm100
    return sm100


def _ref():
    from nanoengine_b200.ops import reference
    return reference


def rel(a, b):
    return float((a.float().cpu() - b.float().cpu()).abs().max() / b.float().abs().max().clamp_min(1e-6))


# ---- kernels -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 8, 64), (3, 96, 72), (70, 136, 128), (129, 64, 200), (128, 520, 4096), (300, 4104, 512), (5, 97, 76)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_bias_is_added_before_the_rounding(M, N, K, dtype):
    k = _k()
    g = torch.Generator(device=DEV).manual_seed(M)
    x, w = torch.randn(M, K, generator=g, device=DEV).to(dtype), torch.randn(N, K, generator=g, device=DEV).to(dtype)
    b = 40 * torch.randn(N, generator=g, device=DEV)
    want = x.double() @ w.double().T + b.double()
    assert rel(k.linear(x, w, None, b), want) < (5e-6 if dtype == torch.float32 else 4.1e-3)
    assert rel(k.linear(x, w, None, b, out_fp32=True), want) < (5e-6 if dtype == torch.float32 else 1e-5)


@pytest.mark.parametrize("T,W,S", [(1, 76, 3), (5, 128, 2), (33, 320, 1), (4, 4096, 4), (2, 20000, 2), (3, 64, 5), (2, 50, 16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_streams(T, W, S, dtype):
    k, r = _k(), _ref()
    g = torch.Generator(device=DEV).manual_seed(T + W)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    y = (3 * rnd(T, W + 4)).to(dtype)[:, :W]
    x, wo, wi, mix, wn = rnd(T, S, W), rnd(S), rnd(S), rnd(S, S), (1 + 0.3 * rnd(W)).to(dtype)
    hw, xw = r.stream_mix(y.float(), x.clone(), wo, mix, wi, wn, 1e-3)
    h, x2 = k.stream_mix(y, x.clone(), wo, mix, wi, wn, 1e-3)
    tol = 5e-6 if dtype == torch.float32 else 5e-3
    assert rel(x2, xw) < 2e-6 and rel(h, hw) < tol
    keep = x.clone()
    h, x3 = k.stream_mix(y, keep, wo, mix, wi, wn, 1e-3, last=True)
    assert rel(h, hw) < tol and torch.equal(x3, x)
    table, pos = rnd(11, W).to(dtype), rnd(9, W).to(dtype)
    ids, at = torch.randint(0, 11, (T,), generator=g, device=DEV), torch.randint(0, 9, (T,), generator=g, device=DEV)
    for p in (pos, None):
        h, x0 = k.stream_embed(ids, at, table, p, wi, wn, 1e-3)
        hw, xw = r.stream_embed(ids, at, table.float(), None if p is None else p.float(), wi, wn, 1e-3)
        assert torch.equal(x0, xw) and rel(h, hw) < tol


@pytest.mark.parametrize("I", [50, 256, 384])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_clamped_linear_activation_and_caps(I, dtype):
    x = (2 * torch.randn(7, 2 * I, device=DEV)).to(dtype)
    act = ("clamp_linear", 1.3, 1.702)
    assert rel(_k().silu_and_mul(x, act=act), _ref().silu_and_mul(x.float(), act=act)) < (2e-6 if dtype == torch.float32 else 5e-3)
    z = 30 * torch.randn(5, I, device=DEV)
    assert rel(_k().cap_logits(z.clone(), 12.5), _ref().cap_logits(z, 12.5)) < 1e-6


@pytest.mark.parametrize("G,D,Dv", [(2, 12, 20), (2, 32, 48), (1, 9, 7), (4, 128, 128)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_kv_rows(G, D, Dv, dtype):
    T = 9
    p = torch.randn(T, 8 + G * (D + Dv), device=DEV).to(dtype)
    k, v = p[:, 8: 8 + G * D], p[:, 8 + G * D:]
    slots = torch.randperm(128, device=DEV)[:T]
    slots[3] = -1
    got = [torch.full((2, 64, G, w), 7.0, device=DEV, dtype=dtype) for w in (D, Dv)]
    want = [t.clone() for t in got]
    _k().kv_rows(*got, slots, k, v)
    _ref().kv_rows(*want, slots, k, v)
    assert all(torch.equal(a, b) for a, b in zip(got, want))


def _paged(q_lens, ctx, G, D, Dv, dtype, g):
    pages = [(c + 63) // 64 for c in ctx]
    perm = torch.randperm(sum(pages) + 3, generator=g, device=DEV)
    bt = torch.zeros(len(ctx), max(pages), dtype=torch.int32, device=DEV)
    at = 0
    for i, n in enumerate(pages):
        bt[i, :n] = perm[at: at + n].int()
        at += n
    kc, vc = (torch.randn(sum(pages) + 3, 64, G, w, generator=g, device=DEV).to(dtype) for w in (D, Dv))
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32, device=DEV)
    return kc, vc, bt, cu, torch.tensor(ctx, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 56, 40), (6, 2, 80, 24), (8, 8, 128, 128), (32, 4, 128, 64), (5, 1, 64, 256), (24, 2, 256, 200), (128, 1, 72, 8),
                                      (7, 7, 8, 16), (3, 1, 12, 20), (10, 2, 17, 5)])
@pytest.mark.parametrize("window,cap,biased", [(0, 0.0, False), (70, 14.0, True), (64, 0.0, True), (1, 30.0, False), (129, 5.0, True)])
@pytest.mark.parametrize("q_lens,ctx", [([1, 1, 1], [1, 64, 700]), ([5, 130, 1, 33], [5, 200, 129, 95])])
def test_biased_attention(H, G, D, Dv, window, cap, biased, q_lens, ctx):
    """Pages in shuffled order against the 32-bit statement, on the tensor cores where the sizes allow it and on the generic kernel; one key of
    each sequence stands out just inside the window of its last query, another one just outside."""
    from nanoengine_b200.ops import sm100_attn
    for dtype in (torch.bfloat16, torch.float32):
        g = torch.Generator(device=DEV).manual_seed(H + D)
        T = sum(q_lens)
        kc, vc, bt, cu, cl = _paged(q_lens, ctx, G, D, Dv, dtype, g)
        p = torch.randn(T, H * D + (8 - H * D % 8) % 8 + (H + 7) // 8 * 8, generator=g, device=DEV).to(dtype)
        q, gate = p[:, : H * D].unflatten(-1, (H, D)), p[:, -((H + 7) // 8 * 8):][:, :H]
        row = 0
        for i, n in enumerate(q_lens):
            row += n
            for d in (window - 1, window) if window else (ctx[i] // 2,):
                j = ctx[i] - 1 - d
                if 0 <= j and d > 0:
                    kc[bt[i, j // 64], j % 64, (H // 2) // (H // G)] = q[row - 1, H // 2] * 0.5
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], device=DEV) if biased else None
        want = _ref().gqa_attention_biased(q.float(), kc.float(), vc.float(), bt, cu, cl, 1.3 * D ** -0.5, window, cap, slopes, gate.float(), 0.7)
        on_tc = dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0
        for splits in (None, 1, 3) if on_tc else (None,):
            y = torch.zeros(T, H * Dv + 8, device=DEV, dtype=dtype)
            before = sm100_attn.BIASED_TC_CALLS[0]
            sm100_attn.gqa_attention_biased(q, kc, vc, bt, cu, cl, 1.3 * D ** -0.5, window, cap, slopes, gate, 0.7, y[:, : H * Dv], max(q_lens), splits)
            assert sm100_attn.BIASED_TC_CALLS[0] == before + int(on_tc)
            assert rel(y[:, : H * Dv], want) < (1e-2 if dtype == torch.bfloat16 else 5e-6), (dtype, splits)
            assert float(y[:, H * Dv:].abs().max()) == 0.0
    assert _k().kernel_status()[0] == 0


LENS = [([1, 1, 1], [0, 0, 1]), ([37, 1, 2, 9], [1, 0, 0, 1]), ([2, 1], [0, 0]), ([8, 16, 17], [0, 1, 0]), ([200, 1, 129], [0, 0, 1])]


def _cu(lens):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)


def _mamba_case(H, G, Dv, N, K, parts, lens, fresh, dtype, seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    T, B, inner, C = sum(lens), len(lens), H * Dv, H * Dv + 2 * G * N
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    return dict(proj=rnd(T, inner + C).to(dtype), dt_raw=rnd(T, H + 3)[:, :H], conv_w=(0.5 * rnd(C, K)).to(dtype), conv_b=(0.3 * rnd(C)).to(dtype), A_log=0.7 * rnd(H),
                dt_bias=rnd(H) - 2, D=rnd(H), norm_w=(1 + 0.2 * rnd(inner)).to(dtype), norm_groups=parts, window=rnd(B + 2, K - 1, C).to(dtype),
                state=0.3 * rnd(B + 2, H, Dv, N), slots=torch.randperm(B + 2, generator=g, device=DEV)[:B].int(), cu_seqlens=_cu(lens),
                fresh=torch.tensor(fresh, dtype=torch.int32, device=DEV), H=H, G=G, Dv=Dv, N=N, eps=1e-4, max_q_len=max(lens))


@pytest.mark.parametrize("H,G,Dv,N,K,parts", [(6, 3, 10, 14, 3, 4), (6, 1, 40, 56, 3, 1), (8, 2, 32, 64, 4, 2), (3, 1, 24, 144, 5, 3), (4, 4, 88, 16, 1, 1), (8, 8, 16, 128, 9, 8),
                                              (16, 2, 64, 128, 4, 16), (2, 1, 160, 40, 2, 1), (1, 1, 33, 300, 4, 1), (4, 1, 64, 256, 16, 2)])
@pytest.mark.parametrize("lens,fresh", LENS)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mamba2_mix(H, G, Dv, N, K, parts, lens, fresh, dtype):
    c = _mamba_case(H, G, Dv, N, K, parts, lens, fresh, dtype)
    want = {n: (v.clone() if isinstance(v, torch.Tensor) else v) for n, v in c.items()}      # the statement rounds where the kernels do
    out, ref_out = _k().mamba2_mix(**c), _ref().mamba2_mix(**want)
    tol = 3e-5 if dtype == torch.float32 else 1.2e-2
    assert rel(c["state"], want["state"]) < tol and torch.equal(c["window"], want["window"])
    assert rel(out, ref_out) < tol
    assert _k().kernel_status()[0] == 0


def _lightning_case(H, Dk, Dv, lens, fresh, dtype, seed=0, decay=None):
    g = torch.Generator(device=DEV).manual_seed(seed)
    T, B = sum(lens), len(lens)
    p = torch.randn(T, 2 * H * Dk + 2 * H * Dv, generator=g, device=DEV).to(dtype)
    q, k, v, gate = p.split([H * Dk, H * Dk, H * Dv, H * Dv], -1)
    decay = torch.tensor(decay if decay else [1 - 0.5 ** (1 + 9 * h / H) for h in range(H)], device=DEV)
    return dict(q=q, k=k, v=v, gate=gate, decay=decay, norm_w=(1 + 0.2 * torch.randn(H * Dv, generator=g, device=DEV)).to(dtype),
                state=0.3 * torch.randn(B + 2, H, Dv, Dk, generator=g, device=DEV), slots=torch.randperm(B + 2, generator=g, device=DEV)[:B].int(), cu_seqlens=_cu(lens),
                fresh=torch.tensor(fresh, dtype=torch.int32, device=DEV), H=H, Dk=Dk, Dv=Dv, eps=1e-4, out_scale=0.6, max_q_len=max(lens))


@pytest.mark.parametrize("H,Dk,Dv,decay", [(3, 10, 14, None), (4, 64, 24, None), (2, 128, 128, None), (4, 24, 8, [0.0, 0.5, 0.99, 1.0]), (8, 16, 64, None), (1, 72, 16, [0.9]),
                                           (2, 17, 5, None), (2, 200, 96, None), (16, 128, 64, None)])
@pytest.mark.parametrize("lens,fresh", LENS)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_lightning_mix(H, Dk, Dv, decay, lens, fresh, dtype):
    c = _lightning_case(H, Dk, Dv, lens, fresh, dtype, decay=decay)
    want = {n: (v.clone() if isinstance(v, torch.Tensor) else v) for n, v in c.items()}
    T = sum(lens)
    y = torch.zeros(T, 8 + H * Dv, device=DEV, dtype=dtype)
    _k().lightning_mix(**c, out=y[:, 8:])
    ref_out = _ref().lightning_mix(**want)
    tol = 3e-5 if dtype == torch.float32 else 1.2e-2
    assert rel(c["state"], want["state"]) < tol and rel(y[:, 8:], ref_out) < tol and float(y[:, :8].abs().max()) == 0.0
    assert _k().kernel_status()[0] == 0


@pytest.mark.parametrize("H,Hk,Dk,Dv", [(4, 4, 64, 64), (2, 1, 128, 128), (3, 3, 48, 40), (2, 2, 8, 200), (8, 2, 120, 64)])
@pytest.mark.parametrize("lens,fresh", [([128], [1]), ([64], [0]), ([129, 40, 31, 1], [0, 1, 0, 0]), ([1000, 2, 255], [1, 1, 0])])
def test_chunked_recurrence_on_tensor_cores(H, Hk, Dk, Dv, lens, fresh):
    """The chunked form against the token-by-token statement in 64-bit: head and remainder of every fp32 operand keep it near 32-bit accuracy,
    for decays from none to complete."""
    k, r = _k(), _ref()
    g = torch.Generator(device=DEV).manual_seed(H * Dk)
    T, B = sum(lens), len(lens)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    qkv = rnd(T, 2 * Hk * Dk + H * Dv).to(torch.bfloat16)
    q, kk, v = qkv.split([Hk * Dk, Hk * Dk, H * Dv], -1)
    log_a = -torch.exp(3 * rnd(T, H)) * 0.05
    log_a[:, 0] = 0.0
    if T > 70:
        log_a[33:70:9] = -300.0
    b = rnd(T, H).abs()
    gates, skip = torch.stack([log_a, b], -1).contiguous(), rnd(H)
    state = 0.3 * rnd(B + 1, H, Dv, Dk)
    want_s, slots, cu, fr = state.double(), torch.randperm(B + 1, generator=g, device=DEV)[:B].int(), _cu(lens), torch.tensor(fresh, dtype=torch.int32, device=DEV)
    rep = H // Hk
    dbl = lambda t, h, d: t.double().reshape(T, h, d)
    want = r._decay_ragged(dbl(q, Hk, Dk).repeat_interleave(rep, 1), dbl(kk, Hk, Dk).repeat_interleave(rep, 1), dbl(v, H, Dv), log_a.double(), b.double(), want_s, slots, cu, fr,
                           skip.double())
    raw = torch.full((T, H * Dv), 9.0, device=DEV)
    before = k.CHUNKED_CALLS[0]
    k._decay_scan(q, kk, v, gates, None, skip, state, slots, cu, fr, raw, H, Hk, Dk, Dv, 0, max(lens))
    assert k.CHUNKED_CALLS[0] == before + 1 and k.kernel_status()[0] == 0
    scale = lambda t: t.abs().max()
    assert float((raw.view(T, H, Dv).double() - want).abs().max() / scale(want)) < 4e-5
    assert float((state.double() - want_s).abs().max() / scale(want_s)) < 4e-5


@pytest.mark.parametrize("which", ["mamba2", "lightning"])
def test_recurrences_do_not_depend_on_the_cut(which):
    n = 300
    c = _mamba_case(8, 2, 64, 64, 4, 2, [n], [1], torch.bfloat16) if which == "mamba2" else _lightning_case(4, 64, 64, [n], [1], torch.bfloat16)
    fn = _k().mamba2_mix if which == "mamba2" else _k().lightning_mix
    whole = {k: (v.clone() if isinstance(v, torch.Tensor) else v) for k, v in c.items()}
    out = fn(**whole)
    at, got = 0, []
    rows = ("proj", "dt_raw") if which == "mamba2" else ("q", "k", "v", "gate")
    for m in (1, 2, 33, 1, 1, 128, 65, 2, 67):
        part = dict(c, cu_seqlens=_cu([m]), fresh=torch.tensor([int(at == 0)], dtype=torch.int32, device=DEV), max_q_len=m, **{r: c[r][at: at + m] for r in rows})
        got.append(fn(**part))
        at += m
    assert at == n and rel(c["state"], whole["state"]) < 1e-4 and rel(torch.cat(got), out) < 5e-3


# ---- the engine ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_engine_agrees_with_the_oracle(name, dtype, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=4.0 if dtype == "float32" else 1.5)
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


def test_long_decoding(tmp_path):
    """Several hundred single tokens through the decode graph: states, windows and pages carried all the way."""
    cfg, W, path = build("mamba_first", tmp_path, sharp=3.0)
    toks = tokens(500, cfg["vocab"], 8)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", DEV, pages=8)
    assert error(feed_all(llm, None, toks, [20, 1]), want) < TOL["float32"]


def test_pool_sized_from_the_free_memory(tmp_path):
    """The start-up pass that measures activations uses the whole token budget, several sequences of it where the learned positions end earlier."""
    from nanoengine_b200 import LLM, Config, SamplingParams
    cfg, W, path = build("odd", tmp_path)
    llm = LLM(Config(model=path, dtype="bfloat16", device=DEV, max_num_seqs=4, max_num_batched_tokens=1000, gpu_memory_utilization=0.05, executor_backend="inproc",
                     enable_prefix_caching=False, status_log_interval_s=0))
    assert llm.engine.scheduler.num_free_blocks(0) > 100
    out = llm.generate([tokens(70, cfg["vocab"], 1)], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(out[0]["token_ids"]) == 4 and _k().kernel_status()[0] == 0
