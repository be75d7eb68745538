"""Tuvutar on the GPU: every kernel against its 32-bit PyTorch statement, and the engine - prompts, portions, mixed batches, decode
graphs, generation - against the plain oracle, in true 32-bit and in bf16."""
import pytest
import torch

import tuvutar_oracle as oracle
from tuvutar_models import CONFIGS, build, error, feed_all, make_llm, tokens

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {"float32": 5e-5, "bfloat16": 0.08}


def _k():
    from nanoengine_b200.ops import sm100
    return sm100


def _ref():
    from nanoengine_b200.ops import reference
    return reference


def rel(a, b):
    return float((a.float().cpu() - b.float().cpu()).abs().max() / b.float().abs().max().clamp_min(1e-6))


# ---- kernels -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 7, 5), (3, 97, 76), (70, 130, 33), (129, 64, 200)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_simt_gemm(M, N, K, dtype):
    k = _k()
    g = torch.Generator(device=DEV).manual_seed(M)
    x = torch.randn(M, K + 3, generator=g, device=DEV).to(dtype)[:, :K]
    w = torch.randn(N, K, generator=g, device=DEV).to(dtype)
    want = x.double() @ w.double().T
    assert rel(k._linear_simt(x, w, None, False), want) < (2e-6 if dtype == torch.float32 else 6e-3)
    assert rel(k.linear_fp32(x, w), want) < (2e-6 if dtype == torch.float32 else 1e-5)
    H, A, B = 3, K, N
    xs = torch.randn(M, H * A + 1, generator=g, device=DEV).to(dtype)[:, : H * A].unflatten(-1, (H, A))
    wb = torch.randn(H, A, B, generator=g, device=DEV).to(dtype)
    out = torch.zeros(M, H, B + 5, device=DEV, dtype=dtype)
    k.bmm_absorb(xs, wb, out=out[..., :B])
    assert rel(out[..., :B], torch.einsum("tha,hab->thb", xs.double(), wb.double())) < (2e-6 if dtype == torch.float32 else 6e-3)
    assert float(out[..., B:].abs().max()) == 0.0


@pytest.mark.parametrize("T,W", [(1, 76), (5, 128), (33, 320), (4, 4096), (2, 20000)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_residual_norm(T, W, dtype):
    k, r = _k(), _ref()
    g = torch.Generator(device=DEV).manual_seed(T + W)
    y = (3 * torch.randn(T, W + 4, generator=g, device=DEV)).to(dtype)[:, :W]
    x = torch.randn(T, W, generator=g, device=DEV)
    wp, wn = ((0.3 * torch.randn(W, generator=g, device=DEV)).to(dtype) for _ in range(2))
    for off in (True, False):
        hw, xw = r.residual_norm(y.float(), x.clone(), wp, wn, 1e-3, off)
        h, x2 = k.residual_norm(y, x.clone(), wp, wn, 1e-3, off)
        assert rel(x2, xw) < 2e-6 and rel(h, hw) < (4e-6 if dtype == torch.float32 else 5e-3)
    table = torch.randn(11, W, generator=g, device=DEV).to(dtype)
    ids = torch.randint(0, 11, (T,), generator=g, device=DEV)
    h, x0 = k.embed_norm(ids, table, wn, 1e-3)
    hw, xw = r.embed_norm(ids, table.float(), wn, 1e-3)
    assert torch.equal(x0, xw) and rel(h, hw) < (4e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("I", [50, 320, 96])
@pytest.mark.parametrize("act", [None, ("gelu_tanh",), ("clamp", 1.5), ("situ", 4.0, 25.0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_activation_of_any_width(I, act, dtype):
    x = (2 * torch.randn(7, 2 * I, device=DEV)).to(dtype)
    assert rel(_k().silu_and_mul(x, act=act), _ref().silu_and_mul(x.float(), act=act)) < (2e-6 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("H,nope,rope,R", [(3, 12, 4, 28), (8, 32, 16, 64), (1, 40, 8, 72)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_prepare(H, nope, rope, R, dtype):
    k, r = _k(), _ref()
    T = 9
    a = torch.randn(T, H * (nope + rope) + R + rope, device=DEV).to(dtype)
    w = torch.randn(R, device=DEV).to(dtype)
    table = r.rope_cos_sin_cache(rope, 4000, 300.0).to(DEV)
    pos = torch.randint(0, 4000, (T,), device=DEV)
    slots = torch.randperm(128, device=DEV)[:T]
    slots[3] = -1
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    for kv in (True, False):
        for full in (True, False):
            q = a[:, : H * (nope + rope)].clone().unflatten(-1, (H, nope + rope))
            kva = a[:, H * (nope + rope):] if kv else None
            cache = torch.full((2, 64, R + rope), 7.0, device=DEV, dtype=dtype)
            want_c, qf, qw = cache.float().clone(), q.float().clone(), torch.zeros(T, H, R + rope, device=DEV)
            got_f = torch.zeros(T, H, R + rope, device=DEV, dtype=dtype)
            k.latent_prepare(q, nope, kva, w if kv else None, 1e-3, pos, table, cache, slots, R, got_f if full else None)
            r.latent_prepare(qf, nope, kva.float() if kv else None, w.float() if kv else None, 1e-3, pos, table, want_c, slots, R, qw if full else None)
            assert rel(q, qf) < tol and rel(cache, want_c) < tol
            if full:
                assert rel(got_f, qw) < tol and float(got_f[..., :R].abs().max()) == 0.0
    if dtype == torch.bfloat16 and (R + rope) % 8 == 0:
        rows = k.latent_gather(cache, slots)
        assert torch.equal(rows, cache.view(-1, R + rope)[slots.clamp_min(0)])


def _delta_case(Hk, Hv, Dk, Dv, K, lens, fresh, dtype, seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    T, C, B = sum(lens), 2 * Hk * Dk + Hv * Dv, len(lens)
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    proj = rnd(T, C + Hv * Dv + 3).to(dtype)[:, : C + Hv * Dv]
    if dtype == torch.bfloat16:
        proj = proj.contiguous()
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)
    return dict(proj=proj, ab=rnd(T, 2 * Hv), conv_w=(0.5 * rnd(C, K)).to(dtype), A_log=0.3 * rnd(Hv), dt_bias=0.5 * rnd(Hv) - 2, norm_w=rnd(Dv).to(dtype),
                window=rnd(B + 2, K - 1, C).to(dtype), state=0.2 * rnd(B + 2, Hv, Dv, Dk), slots=torch.randperm(B + 2, generator=g, device=DEV)[:B].int(),
                cu_seqlens=cu, fresh=torch.tensor(fresh, dtype=torch.int32, device=DEV), Hk=Hk, Hv=Hv, Dk=Dk, Dv=Dv, eps=1e-4, max_q_len=max(lens))


@pytest.mark.parametrize("Hk,Hv,Dk,Dv,K", [(2, 6, 10, 14, 3), (4, 4, 36, 18, 2), (4, 8, 64, 32, 4), (1, 2, 128, 128, 4), (1, 3, 144, 24, 5), (1, 1, 16, 88, 4),
                                           (5, 5, 24, 8, 6), (2, 2, 96, 160, 4), (1, 2, 256, 40, 1), (1, 1, 300, 33, 4), (2, 4, 80, 128, 9), (16, 32, 32, 64, 4)])
@pytest.mark.parametrize("lens,fresh", [([1, 1, 1], [0, 0, 1]), ([37, 1, 2, 9], [1, 0, 0, 1]), ([2, 1], [0, 0]), ([8, 16, 17], [0, 1, 0])])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_delta(Hk, Hv, Dk, Dv, K, lens, fresh, dtype):
    c = _delta_case(Hk, Hv, Dk, Dv, K, lens, fresh, dtype)
    want = {n: (v.float().clone() if isinstance(v, torch.Tensor) and v.is_floating_point() else v) for n, v in c.items()}
    out = _k().gated_delta(**c)
    ref_out = _ref().gated_delta(**want)
    assert rel(c["state"], want["state"]) < 2e-5
    assert torch.equal(c["window"].float(), want["window"])
    assert rel(out, ref_out) < (5e-5 if dtype == torch.float32 else 8e-3)


def test_gated_delta_does_not_depend_on_the_cut():
    c = _delta_case(2, 4, 64, 64, 4, [70], [1], torch.bfloat16)
    whole = {n: (v.clone() if isinstance(v, torch.Tensor) else v) for n, v in c.items()}
    out = _k().gated_delta(**whole)
    at, got = 0, []
    for n in (1, 2, 33, 1, 1, 32):
        part = dict(c, proj=c["proj"][at: at + n], ab=c["ab"][at: at + n], cu_seqlens=torch.tensor([0, n], dtype=torch.int32, device=DEV),
                    fresh=torch.tensor([int(at == 0)], dtype=torch.int32, device=DEV), max_q_len=n)
        got.append(_k().gated_delta(**part))
        at += n
    assert rel(c["state"], whole["state"]) < 1e-6 and torch.equal(c["window"], whole["window"]) and rel(torch.cat(got), out) < 5e-3


@pytest.mark.parametrize("H,R,rope", [(3, 56, 8), (6, 128, 16), (8, 64, 16), (16, 96, 32), (32, 256, 64), (40, 320, 64), (16, 512, 64), (128, 512, 64),
                                      (100, 72, 8), (200, 64, 64), (1, 448, 24)])
@pytest.mark.parametrize("q_lens,ctx", [([1, 1, 1], [1, 64, 700]), ([5, 130, 1, 33], [5, 200, 129, 95])])
def test_latent_attention_on_tensor_cores(H, R, rope, q_lens, ctx):
    """bf16 pages in shuffled order against the 32-bit statement; one key of each sequence is made to stand out."""
    from nanoengine_b200.ops import sm100_attn
    g = torch.Generator(device=DEV).manual_seed(H + R)
    D, T, B = R + rope, sum(q_lens), len(q_lens)
    pages = [(c + 63) // 64 for c in ctx]
    perm = torch.randperm(sum(pages) + 3, generator=g, device=DEV)
    bt = torch.zeros(B, max(pages), dtype=torch.int32, device=DEV)
    cache = torch.randn(sum(pages) + 3, 64, D, generator=g, device=DEV).to(torch.bfloat16)
    q = torch.randn(T, H, D, generator=g, device=DEV).to(torch.bfloat16)
    at, row = 0, 0
    for i, n in enumerate(pages):
        bt[i, :n] = perm[at: at + n].int()
        far = ctx[i] // 3
        cache[bt[i, far // 64], far % 64] = q[row + q_lens[i] - 1, H // 2] * 0.5
        at, row = at + n, row + q_lens[i]
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32, device=DEV)
    cl = torch.tensor(ctx, dtype=torch.int32, device=DEV)
    want = _ref().mla_attention_paged(q.float(), cache.float(), bt, cu, cl, D ** -0.5, R)
    for splits in (None, 1, 3):
        before = sm100_attn.LATENT_TC_CALLS[0]
        got = sm100_attn.mla_attention_paged(q, cache, bt, cu, cl, D ** -0.5, R, splits=splits, max_q_len=max(q_lens))
        assert sm100_attn.LATENT_TC_CALLS[0] == before + 1
        assert rel(got, want) < 1e-2, splits
    assert _k().kernel_status()[0] == 0


def test_generic_attention_in_32_bit():
    g = torch.Generator(device=DEV).manual_seed(1)
    H, R, rope = 5, 28, 4
    cache = torch.randn(4, 64, R + rope, generator=g, device=DEV)
    q = torch.randn(7, H, R + rope, generator=g, device=DEV)
    bt = torch.tensor([[2, 0, 3], [1, 1, 1]], dtype=torch.int32, device=DEV)
    cu, cl = torch.tensor([0, 6, 7], dtype=torch.int32, device=DEV), torch.tensor([150, 1], dtype=torch.int32, device=DEV)
    assert rel(_k().mla_attention_paged(q, cache, bt, cu, cl, 0.3, R), _ref().mla_attention_paged(q, cache, bt, cu, cl, 0.3, R)) < 3e-6


# ---- the engine ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_engine_agrees_with_the_oracle(name, dtype, tmp_path):
    cfg, W, path = build(name, tmp_path, sharp=4.0 if dtype == "float32" else 1.5)
    toks = tokens(200, cfg["vocab"], 1)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, dtype, DEV, pages=5)
    for cuts in ([200], [130, 1], [2], [64, 1, 63, 2, 20], [3, 7, 5, 49, 64]):
        assert error(feed_all(llm, None, toks, cuts), want) < TOL[dtype], cuts
    assert llm.engine.scheduler.num_free_blocks(0) == 5
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
        llm = make_llm(path, "float32", DEV, **kw)
        outs = {o["seq_id"]: o["token_ids"] for o in llm.generate(prompts, sp)}
        assert [outs[i + 1] for i in range(len(prompts))] == want, kw
    llm = make_llm(path, "bfloat16", DEV)
    for p in prompts[:3]:
        llm.add_request(p, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for _ in range(6):
        llm.step()
    runner = llm.engine.executor.runner
    assert runner.graphs is not None and runner.graphs.graphs and runner.graph_step_equals_eager()


def test_fp8_latent_rows(tmp_path):
    """Cache rows as e4m3 (an option of the engine): coarse, but the same in one prompt and token by token."""
    cfg, W, path = build("latent_only", tmp_path)
    toks = tokens(130, cfg["vocab"], 5)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "bfloat16", DEV, pages=4, kv_cache_dtype="fp8")
    a, b = feed_all(llm, None, toks, [130]), feed_all(llm, None, toks, [100, 1])
    assert error(a, want) < 0.3 and error(b, a) < 0.1


def test_long_decoding(tmp_path):
    """Several hundred single tokens through the decode graph: states and pages carried all the way."""
    cfg, W, path = build("delta_first", tmp_path, sharp=3.0)
    toks = tokens(500, cfg["vocab"], 8)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "float32", DEV, pages=8)
    assert error(feed_all(llm, None, toks, [20, 1]), want) < TOL["float32"]


def test_expanded_prompts_equal_absorbed_ones(tmp_path):
    """Head sizes the non-absorbed prompt kernel covers: a whole prompt takes it (also in the layer that reads another's rows), a cut
    one does not."""
    from nanoengine_b200.models import deepseek
    import tuvutar_models as M
    cfg = {"architecture": "Tuvutar", "vocab": 160, "width": 256, "norm": {"eps": 1e-6}, "layers": [
        M.latent(4, 128, 64, 128, 192, ff=256, scaling=M.YARN_B), M.delta(4, 2, 128, 128, 4), M.latent(2, 128, 64, 128, 192, src=0, scaling=M.YARN_B)]}
    W = oracle.random_weights(cfg, 2)
    path = M.write_checkpoint(str(tmp_path / "m"), cfg, W)
    toks = tokens(150, 160, 3)
    want = oracle.forward(cfg, W, toks)
    llm = make_llm(path, "bfloat16", DEV, pages=4)
    calls = []
    inner = deepseek.MLAAttention._prefill_nonabsorbed
    deepseek.MLAAttention._prefill_nonabsorbed = lambda self, *a: (calls.append(1), inner(self, *a))[1]
    try:
        assert error(feed_all(llm, None, toks, [150]), want) < TOL["bfloat16"] and len(calls) == 2
        assert error(feed_all(llm, None, toks, [70, 50, 1]), want) < TOL["bfloat16"] and len(calls) == 4
    finally:
        deepseek.MLAAttention._prefill_nonabsorbed = inner
