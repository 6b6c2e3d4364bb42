"""Mubutar on the GPU: each new or extended kernel alone against its plain statement (tests/kernel_refs.py, float64), and
the engine against the plain implementation (tests/plain_mubutar.py) in every way of cutting the work, in float32 and in
bfloat16, through the step function, the trace program and greedy generation."""
import pytest
import torch

import plain_mubutar as P
import tiny
import tiny_mubutar as TM
from kernel_refs import ReferenceKernels

pytestmark = pytest.mark.gpu

REF = ReferenceKernels(torch.float64)
F32_TOL = 5e-5       # times the largest logit: float32 arithmetic against float64
BF16_TOL = 4e-2      # times the largest logit: activations between kernels carry 8 bits, and the tiny models' attention is peaked
BF16_SHARE = 0.7     # of the positions: a bfloat16 rounding can turn an expert choice, which the plain implementation does not follow


def rows_match(out, want, dtype, what="", share=None):
    """float32: every position within F32_TOL of the largest logit.  bfloat16: BF16_SHARE of the positions within BF16_TOL
    of it and the median within three quarters of that (the float32 runs are the sharp test of every mechanism; these show
    that the bfloat16 path computes the same model)."""
    top = max(1.0, float(want.abs().max()))
    err = (out.double() - want.double()).abs().max(dim=-1).values
    if dtype in ("float32", torch.float32):
        bad = ~(err <= F32_TOL * top)
        assert not bool(bad.any()), f"{what}: position {int(bad.nonzero()[0])}: {float(err[bad][0])} > {F32_TOL * top}"
    else:
        good = float((err <= BF16_TOL * top).double().mean())
        assert good >= (share or BF16_SHARE) and float(err.median()) <= 0.75 * BF16_TOL * top, \
            f"{what}: {good:.2f} of the positions within {BF16_TOL * top}, median {float(err.median())}; first look at {int(err.argmax())}"
    return float(err.max())


# (key width, value width) pairs of these tests that the tensor-core attention is compiled for, with and without a cap
CAPPED = ((80, 48), (128, 128), (32, 80), (192, 128), (256, 160), (16, 16), (48, 112))
PLAIN = ((80, 48), (32, 80), (16, 16))


@pytest.fixture(scope="module", autouse=True)
def K():
    from concurrent.futures import ThreadPoolExecutor
    from infurnace_b200.kernels import load_cuda_kernels
    from infurnace_b200.kernels.build import compile_library
    k = load_cuda_kernels()
    jobs = [("attention_mma", k.attention_defines(d, 2, v, True)) for d, v in CAPPED]
    jobs += [("attention_tc", k.attention_defines(d, 2, v, True)) for d, v in CAPPED if d <= 192 and v <= 128]
    jobs += [("attention_mma", k.attention_defines(d, 2, v, False)) for d, v in PLAIN]
    with ThreadPoolExecutor(max_workers=8) as pool:          # what is not there yet, side by side
        list(pool.map(lambda j: compile_library(*j), jobs))
    return k


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol, what=""):
    err = float((got.double().cpu() - want.double().cpu()).abs().max())
    assert err <= tol, f"{what}: {err} > {tol}"


# ------------------------------------------------------------------------------ products with a bias, the scaled embedding
@pytest.mark.parametrize("n,o,k", [(1, 40, 64), (7, 100, 24), (8, 768, 1024), (16, 33, 2048), (40, 520, 320), (64, 256, 4096),
                                   (100, 1000, 512), (300, 264, 96), (2048, 1280, 256), (5, 37, 21)])
@pytest.mark.parametrize("dtype,out_dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
def test_products_with_a_bias(K, n, o, k, dtype, out_dtype):
    """Every route of the product: plain float32, few rows, tcgen05 with one tile per CTA, with the k range shared, odd sizes;
    with and without a unary function after it."""
    g = gen(n * 7 + o)
    x, w, b = torch.randn(n, k, generator=g).to(dtype), (torch.randn(o, k, generator=g) / k ** 0.5).to(dtype), torch.randn(o, generator=g)
    for epilogue in ("none", "relu2"):
        want, got = torch.zeros(n, o, dtype=torch.float64), torch.full((n, o), float("nan"), dtype=out_dtype, device="cuda")
        REF.linear(x, w, want, epilogue=epilogue, bias=b)
        K.linear(x.cuda(), w.cuda(), got, epilogue=epilogue, bias=b.cuda())
        close(got, want, 0.15 if out_dtype == torch.bfloat16 else 1e-4, epilogue)      # a square reaches 30
    K.check_device_errors()


def test_a_bias_after_a_folded_norm(K):
    """The row factor multiplies the product, not the bias; both routes that take a folded norm."""
    for n, o, k in ((4, 96, 256), (30, 200, 512), (100, 512, 1024)):
        g = gen(n)
        a, w1 = torch.randn(n, 64, generator=g).bfloat16(), (torch.randn(k, 64, generator=g) / 8).bfloat16()
        x, nw = torch.randn(n, k, generator=g), 1 + 0.1 * torch.randn(k, generator=g)
        w, b = (torch.randn(o, k, generator=g) / k ** 0.5).bfloat16(), torch.randn(o, generator=g)
        if not (K.can_fold_norm(n, torch.bfloat16, w1.cuda()) and K.can_fold_norm(n, torch.bfloat16, w.cuda())):
            continue
        parts = K.fold_parts(k, n, w1.cuda())
        xg, v, partials = x.cuda(), torch.zeros(n, k, dtype=torch.bfloat16, device="cuda"), torch.zeros(parts, n, device="cuda")
        K.linear_residual_norm(a.cuda(), w1.cuda(), xg, nw.cuda(), v, partials)
        got = torch.zeros(n, o, device="cuda")
        K.linear(v, w.cuda(), got, row_scale=(partials, parts, 1e-5, k), bias=b.cuda())
        xs = x.double() + a.double() @ w1.double().t()
        h = xs / torch.sqrt(xs.pow(2).mean(-1, keepdim=True) + 1e-5) * nw.double()
        close(got, h @ w.double().t() + b.double(), 0.04, f"{n} rows")


def test_embedding_times_a_number(K):
    g = gen(3)
    for dtype in (torch.float32, torch.bfloat16):
        table, ids = torch.randn(50, 36, generator=g).to(dtype), torch.randint(0, 50, (9,), generator=g, dtype=torch.int32)
        want, got = torch.zeros(9, 36), torch.zeros(9, 36, device="cuda")
        REF.embed(table, ids, want, scale=12.5)
        K.embed(table.cuda(), ids.cuda(), got, scale=12.5)
        close(got, want, 1e-5)


# ------------------------------------------------------------------------------ attention alone
def attention_case(g, H, G, D, VD, ps, lens_new, lens_old, dtype, plant=None, spread=1.0, uniform=False):
    """Queries and pages of a step over requests of lens_old + lens_new tokens, pages scattered, what no request owns set to
    a number that would show.  ``plant`` = (distance, request): that request's last query and its key ``distance`` tokens before get
    a score far above the others in every head."""
    total = [a + b for a, b in zip(lens_new, lens_old)]
    pages = [-(-t // ps) for t in total]
    P_ = sum(pages) + 3
    order = torch.randperm(P_, generator=g)[:sum(pages)]
    bt = torch.full((len(total), max(pages) + 1), -1, dtype=torch.int32)
    at = 0
    for r, n in enumerate(pages):
        bt[r, :n] = order[at:at + n]
        at += n
    n = sum(lens_new)
    q = spread * torch.randn(n, H, D, generator=g)
    kp, vp = torch.full((P_, G, ps, D), 30.0), torch.full((P_, G, ps, VD), 30.0)
    for r, t in enumerate(total):
        pos = torch.arange(t)
        page = bt[r].long()[pos // ps]
        kp[page, :, pos % ps] = torch.randn(t, G, D, generator=g)
        vp[page, :, pos % ps] = torch.randn(t, G, VD, generator=g)
    cu = torch.tensor([0] + list(torch.tensor(lens_new).cumsum(0)), dtype=torch.int32)
    if plant is not None:
        dist, r = plant
        p = total[r] - 1 - dist
        row = int(cu[r + 1]) - 1
        mark = torch.randn(G, D, generator=g)
        mark = mark / mark.norm(dim=-1, keepdim=True)
        kp[bt[r, p // ps].long(), :, p % ps] = 8.0 * mark
        q[row] = (12.0 * mark).repeat_interleave(H // G, dim=0)
    seq = torch.tensor(total, dtype=torch.int32)
    q, kp, vp = q.reshape(n, H * D).to(dtype), kp.to(dtype), vp.to(dtype)
    if uniform:                                     # keys and values in one tensor, as the cache keeps streams of one shape
        both = torch.stack((kp, vp), dim=1).contiguous().cuda()
        return q, kp, vp, bt, cu, seq, both[:, 0], both[:, 1]
    return q, kp, vp, bt, cu, seq, kp.cuda(), vp.cuda()


def run_attention(K, case, H, G, D, VD, lens_new, dtype, scale, cap, sink, exact=False, terms=2):
    q, kp, vp, bt, cu, seq, kg, vg = case
    want = torch.zeros(q.shape[0], H * VD, dtype=torch.float64)
    REF.paged_attention_streams(q, H, G, D, VD, kp, vp, bt, cu, seq, want, scale, 0, None, False, softcap=cap, sink=sink)
    got = torch.full((q.shape[0], H * VD), float("nan"), dtype=dtype, device="cuda")
    K.paged_attention_streams(q.cuda(), H, G, D, VD, kg, vg, bt.cuda(), cu.cuda(), seq.cuda(), got, scale, 0, None, False,
                              max_q_len=max(lens_new), max_seq_len=int(seq.max()), min_q_len=min(lens_new), softcap=cap, sink=sink,
                              weight_terms=terms, exact=exact)
    K.check_device_errors()
    return got, want


SHAPES = [(8, 1, 80, 48), (6, 2, 128, 128), (40, 2, 32, 80), (12, 4, 192, 128), (5, 1, 48, 112), (2, 2, 16, 16), (3, 1, 24, 40),
          (10, 2, 256, 160), (32, 1, 128, 128)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,VD", SHAPES)
def test_capped_attention_with_a_sink(K, dtype, H, G, D, VD):
    """Prompts, portions and decoded tokens of unequal requests in one step, pages of 8 to 64; caps that bend most scores, few
    scores and none; no cap; sinks of 0, above and below the scores, none.  The widths cover the tcgen05 and mma.sync kernels
    with TMA and without, groups that do not divide a tile of rows, more than 16 query heads per key head, and the plain kernel."""
    g = gen(H * 1000 + D + VD)
    lens_new, lens_old = [37, 1, 150, 3, 2], [0, 100, 60, 17, 64]
    for ps, cap, sink, spread, uniform in ((16, 4.0, 0.0, 4.0, False), (32, 30.0, 0.0, 1.0, True), (64, 20.0, 2.5, 12.0, False), (16, 55.0, None, 30.0, False),
                                           (8, 5.0, -3.0, 3.0, False), (16, None, 0.0, 2.0, False), (16, 1e6, 0.0, 3.0, False)):
        uniform = uniform and D == VD
        if cap is None and (D, VD) not in PLAIN and D % 16 == 0:
            continue
        case = attention_case(g, H, G, D, VD, ps, lens_new, lens_old, dtype, spread=spread, uniform=uniform)
        got, want = run_attention(K, case, H, G, D, VD, lens_new, dtype, D ** -0.5, cap, sink)
        # bfloat16: the output's own rounding (values reach 4), and where scores reach dozens the few 1e-5 that a score may be off
        close(got, want, 6e-5 if dtype == torch.float32 else 0.018, f"pages of {ps}, cap {cap}, sink {sink}")


def test_capped_attention_takes_the_tensor_core_routes(K):
    """What ran in the cases above: tcgen05 for prompts (value widths to 128, key widths to 192, caps to 60, pages of 16 to 64),
    mma.sync for decoded tokens and the other bfloat16 sizes, the plain kernel for widths that are no multiple of 16."""
    g = gen(1)

    def routes(H, G, D, VD, ps, cap, lens_new, lens_old, exact=False):
        before = (K.tc_attention_calls, K.small_q_calls, K.stream_attention_calls)
        case = attention_case(g, H, G, D, VD, ps, lens_new, lens_old, torch.bfloat16)
        run_attention(K, case, H, G, D, VD, lens_new, torch.bfloat16, 0.2, cap, 0.0, exact=exact)
        return tuple(a - b for a, b in zip((K.tc_attention_calls, K.small_q_calls, K.stream_attention_calls), before))
    assert routes(10, 2, 80, 48, 16, 20.0, [70, 1], [0, 40]) == (1, 1, 0)
    assert routes(10, 2, 80, 48, 16, 20.0, [70, 40], [0, 40]) == (1, 0, 0)
    assert routes(10, 2, 80, 48, 16, 20.0, [1, 1], [9, 40]) == (0, 1, 0)
    assert routes(10, 2, 80, 48, 8, 20.0, [70, 1], [0, 40]) == (0, 1, 0)
    assert routes(10, 2, 80, 48, 16, 80.0, [70, 1], [0, 40]) == (0, 1, 0)
    assert routes(10, 2, 256, 160, 16, 20.0, [70, 1], [0, 40]) == (0, 1, 0)
    assert routes(10, 2, 24, 40, 16, 20.0, [70, 1], [0, 40]) == (0, 0, 1)
    assert routes(10, 2, 80, 48, 16, 20.0, [70, 1], [0, 40], exact=True) == (0, 0, 1)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D,VD,G", [(80, 48, 2), (128, 128, 1), (40, 24, 2)])
@pytest.mark.parametrize("dist", [0, 1, 15, 16, 17, 63, 64, 65, 127, 128, 129, 302, 303])
def test_a_far_key_at_page_and_tile_borders(K, dtype, D, VD, G, dist):
    """One key holds nearly all of the weight of a request's last query: a page's and a tile's first and last place, the
    sequence's first token (303 behind the last of 304), as the last token of a prompt's portion and as a decoded token."""
    H = 8
    for lens_new, lens_old in (([200, 5], [104, 30]), ([1, 5], [303, 30]), ([2, 33], [302, 0]), ([304, 1], [0, 7])):
        g = gen(dist * 31 + D)
        case = attention_case(g, H, G, D, VD, 16, lens_new, lens_old, dtype, plant=(dist, 0))
        got, want = run_attention(K, case, H, G, D, VD, lens_new, dtype, 0.5, 25.0, 0.0)
        close(got, want, 3e-5 if dtype == torch.float32 else 0.018, f"{lens_new} on {lens_old}")
        bt, cu = case[3], case[4]
        p = 303 - dist
        value = case[2][bt[0, p // 16].long(), :, p % 16].repeat_interleave(H // G, dim=0).reshape(-1)
        close(want[int(cu[1]) - 1], value, 0.05, "the planted key holds the weight")


def test_context_divided_among_many_ctas(K):
    """A decoded token over a long context: many splits, the sink joins once; context of one token (the sink holds half)."""
    g = gen(8)
    for H, G, D, VD, lens_new, lens_old in ((16, 2, 80, 48, [1], [5000]), (32, 2, 128, 128, [1, 1, 1], [3000, 0, 17]), (4, 1, 32, 80, [2, 4], [2049, 1])):
        case = attention_case(g, H, G, D, VD, 16, lens_new, lens_old, torch.bfloat16)
        got, want = run_attention(K, case, H, G, D, VD, lens_new, torch.bfloat16, D ** -0.5, 15.0, 3.0)
        close(got, want, 0.012)


def test_padding_requests_get_zeros(K):
    g = gen(9)
    case = list(attention_case(g, 8, 1, 80, 48, 16, [1, 1, 1], [40, 9, 3], torch.bfloat16))
    case[5] = torch.tensor([41, 0, 4], dtype=torch.int32)             # the second is padding: length 0
    got, want = run_attention(K, tuple(case), 8, 1, 80, 48, [1, 1, 1], torch.bfloat16, 0.1, 15.0, 0.0)
    close(got, want, 0.01)
    assert float(got[1].abs().max()) == 0.0


def test_softmax_weights_in_two_terms(K):
    """Every key the same score, so every weight is 1 / (n + 1): with weights of eight bits a constant value would come out off
    by up to 2^-9; with two terms what is left is the rounding of the output.  Prompt and decoded token."""
    H, G, D, VD = 8, 2, 128, 128
    for lens_new, lens_old in (([130], [0]), ([1], [129])):
        g = gen(2)
        q, kp, vp, bt, cu, seq, kg, vg = attention_case(g, H, G, D, VD, 16, lens_new, lens_old, torch.bfloat16)
        q = torch.full_like(q, 1.0)
        kp = torch.full_like(kp, 0.015869140625)
        vp = torch.full_like(vp, 1.0)
        case = (q, kp, vp, bt, cu, seq, kp.cuda(), vp.cuda())
        got, want = run_attention(K, case, H, G, D, VD, lens_new, torch.bfloat16, 1.0, 20.0, 0.0)
        assert torch.equal(got.cpu(), want.to(torch.bfloat16)) or float((got.double().cpu() - want).abs().max()) <= 2.0 ** -9 * 0.51


# ------------------------------------------------------------------------------ experts alone
@pytest.mark.parametrize("E,top,groups,best", [(16, 3, (4, 2), 2), (8, 2, None, 1), (6, 3, (6, 3), 2), (5, 5, None, 2), (64, 6, (8, 3), 2),
                                               (256, 8, (32, 4), 2), (12, 4, (2, 1), 2), (3, 1, (1, 1), 2), (40, 4, (5, 2), 1), (1, 1, None, 2)])
def test_corrected_router(K, E, top, groups, best):
    n = 70
    g = gen(E * 10 + top)
    logits = 2 * torch.randn(n, E, generator=g)
    logits[1] = 0.0                                 # all equal: the lower index among equals, in groups and experts
    logits[2, : E // 2] = 1.0
    for corr, how in ((None, {}), (0.5 * torch.randn(E, generator=g) - 1.5, {}), (0.5 * torch.randn(E, generator=g), dict(weight_scale=2.5)),
                      (torch.randn(E, generator=g), dict(normalise=False))):
        how = {"normalise": True, **how}
        args = dict(experts=E, scoring="sigmoid", groups=groups, group_best=best, **how)
        ids_r, gates_r = torch.zeros(n, top, dtype=torch.int32), torch.zeros(n, top, dtype=torch.float64)
        REF.moe_route(logits, top, ids_r, gates_r, correction=corr, **args)
        ids_g, gates_g = torch.zeros(n, top, dtype=torch.int32, device="cuda"), torch.zeros(n, top, device="cuda")
        cg = corr.cuda() if corr is not None else None
        K.moe_route(logits.cuda(), top, ids_g, gates_g, correction=cg, **args)
        assert torch.equal(ids_g.cpu(), ids_r)
        close(gates_g, gates_r, 2e-6, "weights")
        offs, perm, pos = (torch.zeros(k, dtype=torch.int32, device="cuda") for k in (E + 1, n * top, n * top))
        ids2, gates2 = torch.zeros_like(ids_g), torch.zeros_like(gates_g)
        K.moe_route_plan(logits.cuda(), top, ids2, gates2, offs, perm, pos, correction=cg, **args)
        assert torch.equal(ids2, ids_g) and torch.equal(gates2, gates_g)
    # the plain implementation routes likewise
    c = torch.randn(E, generator=g).double()
    chosen, w = P.route(logits.double(), c, top, groups) if best == 2 else (None, None)
    if chosen is not None:
        K.moe_route(logits.cuda(), top, ids_g, gates_g, experts=E, scoring="sigmoid", groups=groups, group_best=2, normalise=True, correction=c.float().cuda())
        assert torch.equal(ids_g.cpu().long(), chosen)
        close(gates_g, w, 2e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,top,k,o", [(3, 6, 2, 64, 40), (100, 5, 2, 48, 24), (200, 4, 3, 320, 136), (9, 3, 1, 21, 13)])
def test_experts_without_a_gate(K, dtype, n, E, top, k, o):
    g = gen(n + E)
    x, w = torch.randn(n, k, generator=g).to(dtype), (torch.randn(E, o, k, generator=g) / k ** 0.5).to(dtype)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    offs, perm, pos = (torch.zeros(m, dtype=torch.int32) for m in (E + 1, n * top, n * top))
    REF.moe_plan(ids, E, offs, perm, pos)
    for out_dtype in (dtype, torch.float32):
        want, got = torch.zeros(n * top, o, dtype=torch.float64), torch.zeros(n * top, o, dtype=out_dtype, device="cuda")
        REF.moe_linear(x, w, offs, perm, top, want, epilogue="relu2")
        K.moe_linear(x.cuda(), w.cuda(), offs.cuda(), perm.cuda(), top, got, epilogue="relu2")
        close(got, want, 0.1 if out_dtype == torch.bfloat16 else 1e-4)
    if dtype == torch.bfloat16 and K.moe_grouped_tc_ok(n * top, dtype, w.cuda()):
        places = K.moe_padded_rows(n * top, E)
        og, pg, qg, tg = (torch.zeros(m, dtype=torch.int32, device="cuda") for m in (E + 1, places, n * top, places // K.MOE_TILE))
        K.moe_plan_padded(ids.cuda(), E, og, pg, qg, tg)
        xs = torch.zeros(places, k, dtype=dtype, device="cuda")
        K.moe_gather(x.cuda(), pg, top, tg, xs)
        got = torch.zeros(places, o, device="cuda")
        K.moe_linear_grouped(xs, w.cuda(), tg, got, epilogue="relu2")
        close(got[qg.long()], want[pos.long()], 2e-4)
        K.check_device_errors()


@pytest.mark.parametrize("width", [320, 33, 4096, 1028])
def test_combination_into_the_stream_with_the_next_norm(K, width):
    n, top = 11, 3
    g = gen(width)
    y, pos = torch.randn(n * top + 5, width, generator=g), torch.randperm(n * top + 5, generator=g)[:n * top].to(torch.int32)
    gates, x, base, shared = torch.rand(n, top, generator=g), *(torch.randn(n, width, generator=g) for _ in range(3))
    nw = 1 + 0.2 * torch.randn(width, generator=g)
    logit = torch.randn(n, 2, generator=g)
    for b, sh, sl, norm, dtype in ((base, shared, None, True, torch.bfloat16), (base, None, None, True, torch.float32), (None, shared, logit[:, 1], False, None)):
        xr, xg = x.double(), x.cuda()
        out_r = torch.zeros(n, width, dtype=torch.float64) if norm else None
        out_g = torch.zeros(n, width, dtype=dtype, device="cuda") if norm else None
        REF.moe_combine_update(y, pos, gates, xr, base=b, shared=sh, shared_logit=sl, out=out_r, next_weight=nw if norm else None, eps=1e-3)
        slg = logit.cuda()[:, 1] if sl is not None else None
        K.moe_combine_update(y.cuda(), pos.cuda(), gates.cuda(), xg, base=b.cuda() if b is not None else None,
                             shared=sh.cuda() if sh is not None else None, shared_logit=slg, out=out_g,
                             next_weight=nw.cuda() if norm else None, eps=1e-3)
        close(xg, xr, 2e-5, "stream")
        if norm:
            close(out_g, out_r, 2e-5 if dtype == torch.float32 else 0.03, "norm")


# ------------------------------------------------------------------------------ the engine
LENS = [37, 100, 64, 19, 85, 50, 1, 2, 3, 160]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("mubutar"))
    out = {}
    for name in ("M1", "M2", "M3"):
        d = TM.make_model_dir(name, root)
        cfg, w = TM.load_model_dir(d)
        reqs = {f"r{i}": tiny.random_tokens(cfg["vocab"], n, 100 + i) for i, n in enumerate(LENS)}
        out[name] = (d, cfg, w, reqs, {r: P.forward(cfg, w, t).float() for r, t in reqs.items()})
    return out


def _runner(model_dir, name, dtype, pool):
    from infurnace_b200.engine.loading import EngineOptions, build_runner
    ps = TM.TINY[name]["page_size"]
    return build_runner(model_dir, EngineOptions(dtype=dtype, device="cuda", page_size=ps, num_pages=pool // ps, max_num_seqs=4,
                                                 max_num_batched_tokens=pool, max_model_len=pool))[2]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", ["whole", "bulk_tail", "portions", "mixed"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3"])
def test_cutting_modes(models, name, mode, dtype):
    d, cfg, w, reqs, ref = models[name]
    steps = {"whole": tiny.schedule_whole, "bulk_tail": lambda r: tiny.schedule_bulk_tail(r, tail=60),
             "portions": lambda r: tiny.schedule_portions(r, seed=1),
             "mixed": lambda r: tiny.schedule_mixed(r, max_live=4, max_tokens=640, seed=2)}[mode](reqs)
    runner = _runner(d, name, dtype, 640)
    out = tiny.collect(steps, tiny.run_inprocess(runner, steps), cfg["vocab"])
    assert runner.cache.num_free_slots == 4
    assert runner.cache.free_pages() == [g.pool.num_pages for g in runner.cache.kv_groups]
    runner.rt.kernels.check_device_errors()
    if dtype == "float32":
        worst = max(rows_match(out[rid], ref[rid], dtype, f"{name} {mode} {dtype} request {rid}") for rid in reqs)
    else:         # the share of positions is taken over all requests (three of them have one to three tokens)
        worst = rows_match(torch.cat([out[rid] for rid in reqs]), torch.cat([ref[rid] for rid in reqs]), dtype, f"{name} {mode} {dtype}")
    print(f"{name} {mode} {dtype}: worst {worst:.3g} (largest logit {max(float(r.abs().max()) for r in ref.values()):.3g})")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_of_unequal_requests_against_each_alone(models, dtype):
    """The same kernels' results, not the plain implementation's: what else is in the step moves a position by rounding only."""
    d, cfg, w, reqs, _ = models["M3"]
    some = {r: reqs[r] for r in ("r0", "r4", "r7", "r9")}
    alone = tiny.schedule_whole(some)
    a = tiny.collect(alone, tiny.run_inprocess(_runner(d, "M3", dtype, 640), alone), cfg["vocab"])
    together = [{"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in some.items()], "end": list(some)}]
    b = tiny.collect(together, tiny.run_inprocess(_runner(d, "M3", dtype, 640), together), cfg["vocab"])
    for r in some:
        top = max(1.0, float(a[r].abs().max()))
        err = (a[r] - b[r]).abs().max(dim=-1).values
        if dtype == "float32":
            assert float(err.max()) <= F32_TOL * top, r
        else:
            assert float((err <= 0.03 * top).float().mean()) >= 0.8, r        # a rounding can turn an expert choice


def test_the_fast_routes_ran(models):
    """The wider model's bfloat16 steps take the tcgen05 attention and grouped products in prompts, the split attention and the
    folded norms in decoding; its layers would otherwise pass on the plain kernels alone."""
    d, cfg, w, reqs, ref = models["M3"]
    runner = _runner(d, "M3", "bfloat16", 640)
    k = runner.rt.kernels
    runner.use_graphs = False                                      # a replayed graph counts no launches
    before = (k.tc_attention_calls, k.moe_tcgen05_calls, k.stream_attention_calls, k.small_q_calls)
    toks = reqs["r9"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:150], "want": [0]}], "end": []}] + [
        {"step": 1 + i, "entries": [{"id": "a", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks[150:])]
    tiny.run_inprocess(runner, steps)
    assert k.tc_attention_calls - before[0] == 5 and k.moe_tcgen05_calls - before[1] == 4 and k.stream_attention_calls == before[2]
    assert k.small_q_calls - before[3] == 50
    layers = runner.model.layers
    assert layers[4].takes_folded(1) and layers[3].takes_folded(4) and not layers[1].takes_folded(1) and not layers[4].takes_folded(150)


OTHER_SIZES = {
    # widths that are no multiple of 8 (the plain products), heads of 21 and 9, thirteen experts
    "odd": TM.config(53, 100, 1e-5, [
        TM.layer(3, 1, 21, 9, 0.3, 2.0, TM.moe(13, 4, 37, shared=11)), TM.layer(3, 1, 21, 9, 0.3, 5.0, TM.dense(45), kv_from=0),
        TM.layer(6, 2, 20, 30, 0.25, 3.0, TM.moe(15, 3, 20, groups=(5, 3), shared=12))], emb=0.2, logit=2.5),
    # sizes the tensor-core routes take throughout: heads of 128, keys of 192, one key head for 24 query heads, one page's
    # worth of everything; two layers that read in a row
    "tc": TM.config(211, 128, 1e-6, [
        TM.layer(24, 1, 128, 128, 0.09, 30.0, TM.moe(16, 4, 64, groups=(4, 1), shared=64)),
        TM.layer(24, 1, 128, 128, 0.09, 20.0, TM.dense(256), kv_from=0), TM.layer(24, 1, 128, 128, 0.09, 25.0, TM.dense(128), kv_from=0),
        TM.layer(4, 2, 192, 128, 0.07, 45.0, None), TM.layer(4, 4, 16, 16, 0.25, 60.0, TM.moe(8, 2, 32, groups=(2, 2)))], emb=9.0),
    # a single layer with one head; a cap that bends everything; a cap too high for the prompt kernel; no cap
    "one": TM.config(40, 32, 1e-5, [TM.layer(1, 1, 16, 16, 0.3, 0.3, TM.dense(64))], logit=5.0),
    "caps": TM.config(60, 64, 1e-5, [TM.layer(4, 2, 32, 80, 0.2, 300.0, TM.moe(4, 2, 32)), TM.layer(2, 1, 16, 16, 0.3, None, TM.dense(72)),
                                     TM.layer(4, 2, 32, 80, 0.2, 61.0, None, kv_from=0)]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(OTHER_SIZES))
def test_other_sizes_and_orders(tmp_path, name, dtype):
    """Models of other sizes, head counts and orders of layers, in a mixed schedule over a small pool."""
    from infurnace_b200.engine.loading import EngineOptions, build_runner
    conf = OTHER_SIZES[name]
    d = TM.make_model_dir("_" + name, str(tmp_path), config=conf, seed=31, store="bfloat16", sharpen=1.5)
    cfg, w = TM.load_model_dir(d)
    reqs = {f"r{i}": tiny.random_tokens(cfg["vocab"], n, 7 + i) for i, n in enumerate([45, 130, 3, 70, 1, 99, 20])}
    ref = {r: P.forward(cfg, w, t).float() for r, t in reqs.items()}
    steps = tiny.schedule_mixed(reqs, max_live=4, max_tokens=384, seed=3)
    runner = build_runner(d, EngineOptions(dtype=dtype, device="cuda", page_size=16, num_pages=24, max_num_seqs=4,
                                           max_num_batched_tokens=384, max_model_len=384))[2]
    out = tiny.collect(steps, tiny.run_inprocess(runner, steps), cfg["vocab"])
    runner.rt.kernels.check_device_errors()
    assert runner.cache.num_free_slots == 4 and runner.cache.free_pages() == [g.pool.num_pages for g in runner.cache.kv_groups]
    if dtype == "float32":
        for rid in reqs:
            rows_match(out[rid], ref[rid], dtype, f"{name} request {rid}")
    else:
        rows_match(torch.cat([out[r] for r in reqs]), torch.cat([ref[r] for r in reqs]), dtype, name, share=0.6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(models, dtype):
    """Every token alone from the first on, 300 of them."""
    d, cfg, w, _, _ = models["M3"]
    toks = tiny.random_tokens(cfg["vocab"], 300, 77)
    want = P.forward(cfg, w, toks).float()
    steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    out = tiny.collect(steps, tiny.run_inprocess(_runner(d, "M3", dtype, 384), steps), cfg["vocab"])["x"]
    rows_match(out, want, dtype, "token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_in_portions_then_decoding(models, dtype):
    """900 tokens: portions of 500, 133, 2 and 200, then 65 tokens one by one, beside a second request that comes and goes."""
    d, cfg, w, _, _ = models["M3"]
    toks = tiny.random_tokens(cfg["vocab"], 900, 91)
    other = tiny.random_tokens(cfg["vocab"], 90, 92)
    want, want_other = P.forward(cfg, w, toks).float(), P.forward(cfg, w, other).float()
    steps, at = [], 0
    for i, n in enumerate([500, 133, 2, 200] + [1] * 65):
        entries = [{"id": "x", "tokens": toks[at:at + n], "want": list(range(n))}]
        if i == 1:
            entries.append({"id": "y", "tokens": other[:60], "want": list(range(60))})
        if 2 <= i < 32:
            entries.append({"id": "y", "tokens": [other[58 + i]], "want": [0]})
        steps.append({"step": i, "entries": entries, "end": ["y"] if i == 31 else []})
        at += n
    assert at == 900
    out = tiny.collect(steps, tiny.run_inprocess(_runner(d, "M3", dtype, 1088), steps), cfg["vocab"])
    rows_match(out["x"], want, dtype, "the long request")
    rows_match(out["y"], want_other, dtype, "the request beside it")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(models, tmp_path, dtype):
    d, cfg, w, reqs, ref = models["M1"]
    steps = tiny.schedule_mixed(reqs, max_live=4, max_tokens=640, seed=5)
    outputs = tiny.run_trace_run(d, dtype, steps, str(tmp_path / "out"), 640, TM.TINY["M1"]["page_size"])
    out = tiny.collect(steps, outputs, cfg["vocab"])
    rows_match(torch.cat([out[rid] for rid in reqs]), torch.cat([ref[rid] for rid in reqs]), dtype, "all requests")


def test_greedy_generation_through_the_engine_and_its_graphs(models):
    """The engine's own entry point: scheduler, portions beside decoded tokens, six requests over four slots, decode
    steps replayed from CUDA graphs.  In float32 the tokens are the plain implementation's."""
    from infurnace_b200.engine import Engine, EngineOptions, SamplingParams
    d, cfg, w, _, _ = models["M1"]
    ps = TM.TINY["M1"]["page_size"]
    prompts = [tiny.random_tokens(cfg["vocab"], n, 40 + n) for n in (1, 9, 33, 70, 5, 18)]
    want = [P.greedy(cfg, w, p, 16) for p in prompts]
    for graphs in (True, False):
        eng = Engine.from_model_dir(d, EngineOptions(dtype="float32", device="cuda", page_size=ps, num_pages=40, max_num_seqs=4,
                                                     max_num_batched_tokens=32))
        eng.runner.use_graphs = eng.runner.use_graphs and graphs
        assert eng.generate(prompts, SamplingParams(max_tokens=16)) == want
        assert (eng.runner.graph_replays > 0) == graphs
        eng.runner.cache.check()
        assert eng.runner.cache.num_free_slots == 4


def test_bfloat16_graphs_replay_what_eager_steps_compute(models):
    """The wider model's decode steps (folded norms, split attention, grouped experts) give the same tokens replayed or not."""
    from infurnace_b200.engine import Engine, EngineOptions, SamplingParams
    d, cfg, w, _, _ = models["M3"]
    prompts = [tiny.random_tokens(cfg["vocab"], n, 60 + n) for n in (3, 40, 90)]
    outs = []
    for graphs in (True, False):
        eng = Engine.from_model_dir(d, EngineOptions(dtype="bfloat16", device="cuda", page_size=16, num_pages=40, max_num_seqs=4,
                                                     max_num_batched_tokens=64))
        eng.runner.use_graphs = eng.runner.use_graphs and graphs
        outs.append(eng.generate(prompts, SamplingParams(max_tokens=24)))
    assert outs[0] == outs[1]


def test_command_line(models):
    import json
    import os
    import subprocess
    import sys
    d, cfg, w, _, _ = models["M1"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "infurnace-b200"), "--model", d, "--prompt-ids", "5,6,7,8",
                          "--max-tokens", "6", "--json", "--dtype", "float32", "--page-size", "16", "--max-context", "64"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["generated_token_ids"] == P.greedy(cfg, w, [5, 6, 7, 8], 6) and report["model"]["architecture"] == "Mubutar"
