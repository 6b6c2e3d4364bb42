"""Tigelorn on the GPU: each new or extended kernel alone against its plain statement (tests/kernel_refs.py, float64), and
the engine against the plain implementation (tests/plain_tigelorn.py) in every way of cutting the work, in float32 and in
bfloat16, through the step function, the trace program and greedy generation."""
import pytest
import torch

import plain_tigelorn as P
import tiny
import tiny_tigelorn as TT
from kernel_refs import ReferenceKernels

pytestmark = pytest.mark.gpu

REF = ReferenceKernels(torch.float64)
F32_TOL = 5e-5       # times the largest logit: float32 arithmetic against float64
BF16_TOL = 4e-2      # times the largest logit: activations between kernels carry 8 bits, and the tiny models' attention is peaked
BF16_SHARE = 0.9     # of the positions


def rows_match(out, want, dtype, what="", share=None):
    """float32: every position within F32_TOL of the largest logit.  bfloat16: BF16_SHARE of the positions within BF16_TOL
    of it and the median within half of that (the float32 runs are the sharp test of every mechanism; these show that the
    bfloat16 path computes the same model)."""
    top = max(1.0, float(want.abs().max()))
    err = (out.double() - want.double()).abs().max(dim=-1).values
    if dtype in ("float32", torch.float32):
        bad = err > F32_TOL * top
        assert not bool(bad.any()), f"{what}: position {int(bad.nonzero()[0])}: {float(err[bad][0])} > {F32_TOL * top}"
    else:
        good = float((err <= BF16_TOL * top).double().mean())
        assert good >= (share or BF16_SHARE) and float(err.median()) <= 0.5 * BF16_TOL * top, \
            f"{what}: {good:.2f} of the positions within {BF16_TOL * top}, median {float(err.median())}; first look at {int(err.argmax())}"
    return float(err.max())


@pytest.fixture(scope="module")
def K():
    from infurnace_b200.kernels import load_cuda_kernels
    return load_cuda_kernels()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol, what=""):
    err = float((got.double().cpu() - want.double().cpu()).abs().max())
    assert err <= tol, f"{what}: {err} > {tol}"


def requests(lens_new, lens_old=None, pad=0):
    """cu_q, seq_lens, state_slots, req_index (int32) for requests that bring lens_new tokens on top of lens_old; ``pad``
    more requests of length 0 with one row each (the padding of a recorded decode step)."""
    lens_old = lens_old or [0] * len(lens_new)
    cu, req = [0], []
    for r, n in enumerate(lens_new):
        cu.append(cu[-1] + n)
        req += [r] * n
    seq = [a + b for a, b in zip(lens_new, lens_old)]
    for i in range(pad):
        cu.append(cu[-1] + 1)
        seq.append(0)
        req.append(len(lens_new) + i)
    slots = [2 * i + 1 for i in range(len(lens_new))] + [0] * pad       # distinct, out of order with the rows, never slot 0
    return tuple(torch.tensor(v, dtype=torch.int32) for v in (cu, seq, slots, req))


def cuda(*ts):
    return tuple(t.cuda() if t is not None else None for t in ts)


# ------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("vocab,hidden,buckets,mp,mc", [(101, 48, 37, 11, 5), (300, 257, 1, 3, 9), (5000, 64, 4999, 1000003, 2 ** 31 - 1), (50, 33, 7, 0, 1)])
def test_embedding_with_a_pair_table(K, dtype, vocab, hidden, buckets, mp, mc):
    """Several steps over the same slots: the token before a portion comes from the slot, a sequence's first token takes the
    last row; a padding row leaves its slot alone."""
    g = gen(vocab)
    table, pairs = torch.randn(vocab, hidden, generator=g).to(dtype), torch.randn(buckets + 1, hidden, generator=g).to(dtype)
    st_r = torch.full((8, 1), 3.0)
    st_g = st_r.cuda()
    old = [0, 0, 5]
    for step, lens in enumerate(([9, 1, 2], [1, 1, 1], [2, 4, 30], [1, 300, 1])):
        cu, seq, slots, req = requests(lens, old, pad=1 if step == 1 else 0)
        n = int(cu[-1])
        pos = torch.cat([torch.arange(a, a + b) for a, b in zip(old, lens)] + ([torch.zeros(1)] if step == 1 else [])).to(torch.int32)
        ids = torch.randint(0, vocab, (n,), generator=g, dtype=torch.int32)
        out_r, out_g = torch.zeros(n, hidden), torch.zeros(n, hidden, device="cuda")
        REF.embed_bigram(table, pairs, ids, pos, req, cu, seq, slots, st_r, buckets, mp, mc, out_r)
        K.embed_bigram(*cuda(table, pairs, ids, pos, req, cu, seq, slots), st_g, buckets, mp, mc, out_g)
        live = n - (1 if step == 1 else 0)
        close(out_g[:live], out_r[:live], 1e-6, f"step {step}")
        assert torch.equal(st_g.cpu(), st_r), f"step {step}, the tokens kept"
        old = [a + b for a, b in zip(old, lens)]
    K.check_device_errors()


@pytest.mark.parametrize("xd,od", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("n,groups,part", [(7, 3, 40), (5, 1, 33), (300, 1, 256), (9, 1, 257), (4, 2, 3000), (3, 16, 1), (1, 5, 128)])
def test_norm_gate_and_factor_of_rows(K, xd, od, n, groups, part):
    g = gen(n * part)
    width = groups * part
    x = torch.randn(n, width + 5, generator=g).to(xd)
    gate = torch.randn(n, width + 3, generator=g) * 3
    for weight, eps, act, scale, gated in ((torch.randn(width, generator=g), 1e-5, "sigmoid", 1.0, True),
                                           (torch.randn(part, generator=g), 0.3, "silu", -1.7, True),
                                           (None, None, "sigmoid", 0.8, True), (None, 1e-6, "sigmoid", 2.0, False)):
        want = torch.zeros(n, width, dtype=torch.float64)
        wide = torch.full((n, width + 7), 9.0, device="cuda", dtype=od)
        REF.norm_gate_rows(x[:, 5:], want, groups=groups, weight=weight, eps=eps, gate=gate[:, :width] if gated else None, activation=act, scale=scale)
        K.norm_gate_rows(x.cuda()[:, 5:], wide[:, 2:2 + width], groups=groups, weight=weight.cuda() if weight is not None else None, eps=eps,
                         gate=gate.cuda()[:, :width] if gated else None, activation=act, scale=scale)
        close(wide[:, 2:2 + width], want, (2e-5 if od == torch.float32 else 0.01) * max(1.0, float(want.abs().max())), f"{act} {scale}")
        assert float(wide[:, :2].min()) == 9.0 and float(wide[:, 2 + width:].min()) == 9.0        # slices only


DELTA_SIZES = [  # kv_heads, heads, dim, vdim, taps
    (2, 4, 8, 10, 3), (1, 3, 32, 32, 4), (3, 3, 33, 70, 1), (2, 2, 64, 64, 2), (4, 8, 128, 128, 4), (1, 2, 96, 200, 7), (2, 2, 256, 40, 4),
    (1, 1, 130, 129, 3), (1, 2, 260, 24, 2)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,H,D,V,taps", DELTA_SIZES)
def test_delta_convolutions_over_steps_and_slots(K, dtype, G, H, D, V, taps):
    """Several steps over the same slots: portions longer and shorter than the taps' reach, single tokens, a padding row."""
    g = gen(D * 10 + taps)
    C, low_w = 2 * G * D + H * V, 11
    w = torch.randn(C, taps, generator=g)
    st_r = torch.zeros(8, max(taps - 1, 1), C)
    st_g = st_r.cuda()
    old = [0, 0, 0]
    for step, lens in enumerate(([9, 1, 2], [1, 1, 1], [2, taps, 30], [1, 3, 1], [taps + 1, 1, 2], [20, 40, 7])):
        cu, seq, slots, req = requests(lens, old, pad=1 if step == 1 else 0)
        n = int(cu[-1])
        live = n - (1 if step == 1 else 0)
        proj = torch.randn(n, C + H + low_w, generator=g)
        r = [torch.zeros(n, C, dtype=torch.float64), torch.zeros(n, H, dtype=torch.float64), torch.zeros(n, 16, dtype=torch.float64)]
        o = [torch.zeros(n, C, device="cuda"), torch.zeros(n, H, device="cuda"), torch.full((n, 16), 5.0, device="cuda", dtype=dtype)]
        REF.delta_prepare(proj, G, H, D, V, w, 1e-6, st_r, slots, cu, seq, req, *r, low_w)
        K.delta_prepare(proj.cuda(), G, H, D, V, w.cuda(), 1e-6, st_g, *cuda(slots, cu, seq, req), *o, low_w)
        for got, want, tol, what in zip(o, r, (2e-5, 1e-6, 1e-6 if dtype == torch.float32 else 0.02), ("q k v", "beta", "bottlenecks")):
            close(got[:live], want[:live], tol * max(1.0, float(want.abs().max())), f"step {step}, {what}")
        close(st_g, st_r, 1e-6, f"step {step}, the inputs kept")
        old = [a + b for a, b in zip(old, lens)]


def _delta_inputs(g, n, G, H, D, V, spread=2.0):
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q, k = unit(torch.randn(n, G, D, generator=g)) * D ** -0.5, unit(torch.randn(n, G, D, generator=g) + 0.3)
    qkv = torch.cat((q.reshape(n, -1), k.reshape(n, -1), torch.randn(n, H * V, generator=g)), dim=1).contiguous()
    return qkv, torch.randn(n, H * (D + V), generator=g) * spread, torch.rand(n, H, generator=g)


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("G,H,D,V,taps", DELTA_SIZES)
def test_delta_rule_walked_and_in_chunks(K, out_dtype, G, H, D, V, taps):
    """A prompt, portions on top of it and single tokens, decays from almost 1 to almost 0, states that are not zero, slots
    out of order and a padding row; the walk and the chunked form against the same statement."""
    g = gen(D + V)
    rate, bias = torch.exp(torch.linspace(-2.0, 2.5, H)), torch.linspace(-7.0, 4.0, H * D)
    nw = 1 + 0.2 * torch.randn(V, generator=g)
    st_r = torch.randn(8, H, D, V, generator=g)
    st_g = st_r.cuda()
    tol = 1e-4 if out_dtype == torch.float32 else 0.05
    old = [0, 0, 0]
    for step, lens in enumerate(([75, 3, 33], [1, 1, 1], [16, 2, 17], [40, 1, 2], [1, 1, 1])):
        cu, seq, slots, req = requests(lens, old, pad=1 if step in (1, 4) else 0)
        n = int(cu[-1])
        live = n - (1 if step in (1, 4) else 0)
        qkv, up, beta = _delta_inputs(g, n, G, H, D, V)
        out_r, out_g = torch.zeros(n, H * V, dtype=torch.float64), torch.zeros(n, H * V, device="cuda", dtype=out_dtype)
        REF.delta_rule(qkv, up, beta, G, H, D, V, rate, bias, nw, 1e-5, st_r, slots, cu, seq, out_r)
        before = K.delta_chunked_calls
        K.delta_rule(*cuda(qkv, up, beta), G, H, D, V, *cuda(rate, bias, nw), 1e-5, st_g, *cuda(slots, cu, seq), out_g, max_q_len=max(lens))
        assert (K.delta_chunked_calls > before) == (max(lens) >= K.delta_chunk_min and D <= 256)
        close(out_g[:live], out_r[:live], tol * max(1.0, float(out_r.abs().max())), f"step {step}")
        close(st_g, st_r, 3e-5 * max(1.0, float(st_r.abs().max())), f"step {step}, state")
        old = [a + b for a, b in zip(old, lens)]


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("written,read", [(0, 600), (15, 16), (16, 31), (17, 400), (31, 32), (255, 256), (300, 300)])
def test_a_value_written_far_back_is_read(K, written, read, chunked, monkeypatch):
    """One key of its own direction holds a value through hundreds of tokens that do not touch it, read at chunk borders and
    far from them; a second write under that key later replaces it."""
    monkeypatch.setattr(K, "delta_chunk_min", 2 if chunked else 1 << 20)
    g = gen(written * 7 + read)
    G = H = 2
    D = V = 64
    n = 640
    qkv, up, beta = _delta_inputs(g, n, G, H, D, V)
    q, k = qkv[:, :G * D].view(n, G, D), qkv[:, G * D:2 * G * D].view(n, G, D)
    k[..., 0] = 0.0
    k[written] = 0.0
    k[written, :, 0] = 1.0
    if read + 8 < n:
        k[read + 8] = 0.0
        k[read + 8, :, 0] = 1.0
        beta[read + 8] = 1.0
    beta[written] = 1.0
    q[read] = 0.0
    q[read, :, 0] = 1.0
    rate, bias, nw = torch.ones(H), torch.full((H * D,), -40.0), torch.ones(V)             # decays of one
    st = torch.zeros(1, H, D, V)
    cu, seq, slots = (torch.tensor(v, dtype=torch.int32) for v in ([0, n], [n], [0]))
    out = torch.zeros(n, H * V, device="cuda")
    st_g = st.cuda()
    K.delta_rule(*cuda(qkv, up, beta), G, H, D, V, *cuda(rate, bias, nw), 1e-6, st_g, *cuda(slots, cu, seq), out, max_q_len=n)
    v = qkv[written, 2 * G * D:].view(H, V).double()
    want = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + 1e-6) * torch.sigmoid(up[read, H * D:].double().view(H, V))
    close(out[read].view(H, V), want, 1e-4, "the value")
    if read + 8 < n:
        close(st_g[0, :, 0], qkv[read + 8, 2 * G * D:].view(H, V), 1e-4, "the value that replaced it")


@pytest.mark.parametrize("dim,vdim,heads", [(6, 10, 3), (32, 40, 4), (128, 128, 2), (16, 144, 2), (160, 24, 1), (64, 600, 1)])
def test_matrix_state_scan_with_silu_inputs_and_plain_outputs(K, dim, vdim, heads):
    g = gen(dim)
    decay = torch.tensor([0.3, 1.0, 0.99, 0.0])[:heads].contiguous()
    st_r = torch.randn(8, heads, dim, vdim, generator=g)
    st_g = st_r.cuda()
    old = [0, 0]
    for step, lens in enumerate(([150, 3], [1, 1], [30, 98], [1, 2])):
        cu, seq, slots, _ = requests(lens, old, pad=1 if step == 1 else 0)
        n = int(cu[-1])
        live = n - (1 if step == 1 else 0)
        rows = torch.randn(n, heads * (2 * dim + vdim) + 3, generator=g)
        cut = lambda t: (t[:, 3:3 + heads * dim], t[:, 3 + heads * dim:3 + 2 * heads * dim], t[:, 3 + 2 * heads * dim:])
        want, got = torch.zeros(n, heads * vdim, dtype=torch.float64), torch.zeros(n, heads * vdim, device="cuda")
        REF.linear_scan(*cut(rows), None, heads, dim, vdim, st_r, slots, cu, seq, want, 1e-5, decay=decay, activation="silu", finish=False)
        K.linear_scan(*cut(rows.cuda()), None, heads, dim, vdim, st_g, *cuda(slots, cu, seq), got, 1e-5, decay=decay.cuda(),
                      activation="silu", finish=False, max_q_len=max(lens))
        close(got[:live], want[:live], 3e-5 * max(1.0, float(want.abs().max())), f"step {step}")
        close(st_g, st_r, 3e-5 * max(1.0, float(st_r.abs().max())), f"step {step}, state")
        old = [a + b for a, b in zip(old, lens)]


@pytest.mark.parametrize("n,o,k", [(1, 40, 64), (5, 200, 320), (33, 4096, 128), (70, 384, 256), (300, 1024, 512), (9, 24, 30), (128, 8192, 256), (2048, 512, 128)])
def test_products_with_a_gelu_gate(K, n, o, k):
    """On every route of the products (rows, sizes, a folded norm before them), float32 and bfloat16."""
    g = gen(n + o)
    for dtype in (torch.float32, torch.bfloat16):
        x, w = torch.randn(n, k, generator=g).to(dtype), (torch.randn(2 * o, k, generator=g) * (2.0 / k ** 0.5)).to(dtype)
        want, got = torch.zeros(n, o, dtype=torch.float64), torch.zeros(n, o, device="cuda", dtype=dtype)
        REF.linear(x, w, want, epilogue="gelu_gate")
        K.linear(x.cuda(), w.cuda(), got, epilogue="gelu_gate")
        close(got, want, (2e-5 if dtype == torch.float32 else 0.01) * float(want.abs().max()), f"{dtype}")
        if dtype == torch.bfloat16 and K.can_fold_norm(n, dtype, w.cuda(), "silu_gate"):
            partials = torch.rand(2, n, generator=g) * k
            REF.linear(x, w, want, epilogue="gelu_gate", row_scale=(partials, 2, 1e-5, k))
            K.linear(x.cuda(), w.cuda(), got, epilogue="gelu_gate", row_scale=(partials.cuda(), 2, 1e-5, k))
            close(got, want, 0.01 * float(want.abs().max()), "after a folded norm")
    K.check_device_errors()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_store_of_unit_queries_and_keys(K, dtype):
    """q and k heads divided by their root mean square after the rotation, from rows that are a slice of wider ones; with a
    table whose factor is not one (a rotation that changes lengths) the order shows."""
    g = gen(3)
    n, H, G, d, dv, dims, ps = 11, 4, 2, 12, 10, 8, 4
    table = torch.randn(n, dims, generator=g)                      # no rotation at all: lengths change
    wide = torch.randn(n, (H + G) * d + G * dv + 9, generator=g)
    slots = torch.randperm(5 * ps, generator=g)[:n].to(torch.int32)
    slots[2] = -1

    def run(kern, dev, cd, eps):
        q = torch.zeros(n, H * d, dtype=cd, device=dev)
        pk, pv = torch.zeros(5, G, ps, d, dtype=cd, device=dev), torch.zeros(5, G, ps, dv, dtype=cd, device=dev)
        kern.rotary_store(wide.to(dev)[:, :(H + G) * d + G * dv], H, G, d, dv, table.to(dev), dims, False, None, None, False, q, pk, pv,
                          slots.to(dev), qk_eps=eps)
        return q, pk, pv
    for eps in (1e-5, 0.5):
        for got, want, what in zip(run(K, "cuda", dtype, eps), run(REF, "cpu", torch.float64, eps), ("q", "keys", "values")):
            close(got, want, 1e-5 if dtype == torch.float32 else 0.03, what)
    q = run(REF, "cpu", torch.float64, 1e-9)[0].view(n, H, d)
    assert torch.allclose(q.pow(2).mean(-1), torch.ones(n, H, dtype=torch.float64), atol=1e-6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,dv", [(64, 64), (32, 48), (128, 128), (24, 10)])
@pytest.mark.parametrize("window,dist", [(40, 39), (40, 40), (17, 16), (17, 17), (1, 0), (0, 303), (0, 304)])
def test_a_far_key_and_the_windows_edges(K, dtype, d, dv, window, dist):
    """Unit queries and keys over streams of two widths, two-term weights: a planted key that holds all the weight w - 1
    positions behind the last query (just inside the window) and w behind (just outside), far back at a page's first and
    last place without a window; as the last token of a portion and as a single decoded token beside another request."""
    H, G, ps, scale = 4, 2, 16, 24.0 / d
    for lens_new, lens_old in (([50, 20], [270, 3]), ([1, 1], [319, 22])):
        g = gen(window * 7 + dist + d)
        total = [a + b for a, b in zip(lens_new, lens_old)]
        per = [-(-t // ps) for t in total]
        order = torch.randperm(sum(per) + 2, generator=g).tolist()
        bt = torch.full((2, max(per)), -1, dtype=torch.int32)
        pk, pv = torch.zeros(sum(per) + 2, G, ps, d), torch.zeros(sum(per) + 2, G, ps, dv)
        unit = lambda x: x / x.pow(2).mean(-1, keepdim=True).sqrt()
        keys = [unit(torch.randn(t, G, d, generator=g)) for t in total]
        vals = [torch.randn(t, G, dv, generator=g) for t in total]
        q = unit(torch.randn(sum(lens_new), H, d, generator=g))
        row, pos = lens_new[0] - 1, total[0] - 1 - dist
        q[row] = keys[0][pos].repeat_interleave(H // G, dim=0)                   # score 24 against about 0 +- 24 / sqrt(d)
        at = 0
        for i in range(2):
            for j in range(per[i]):
                bt[i, j] = order[at]
                span = slice(j * ps, min((j + 1) * ps, total[i]))
                m = span.stop - span.start
                pk[order[at], :, :m], pv[order[at], :, :m] = keys[i][span].transpose(0, 1), vals[i][span].transpose(0, 1)
                at += 1
        q = q.reshape(-1, H * d)
        q, pk, pv = q.to(dtype), pk.to(dtype), pv.to(dtype)
        cu, seq, _, _ = requests(lens_new, lens_old)
        want, got = torch.zeros(q.shape[0], H * dv, dtype=torch.float64), torch.zeros(q.shape[0], H * dv, device="cuda", dtype=dtype)
        REF.paged_attention_streams(q.double(), H, G, d, dv, pk.double(), pv.double(), bt, cu, seq, want, scale, window, None, False)
        before = K.tc_attention_calls
        K.paged_attention_streams(*cuda(q), H, G, d, dv, *cuda(pk, pv, bt, cu, seq), got, scale, window, None, False,
                                  max_q_len=max(lens_new), max_seq_len=max(total), min_q_len=min(lens_new), weight_terms=2, exact=False,
                                  score_bound=scale * d)
        close(got, want, (2e-5 if dtype == torch.float32 else 0.03) * max(1.0, float(want.abs().max())), f"window {window}, distance {dist}, {lens_new}")
        if dtype == torch.bfloat16 and d % 16 == 0 and max(lens_new) > 1:
            assert K.tc_attention_calls > before                                       # the tcgen05 kernel for bounded scores
        planted = pv[int(bt[0, pos // ps]), :, pos % ps].double().repeat_interleave(H // G, dim=0).reshape(-1)
        inside = window == 0 or dist < window
        if d >= 64:
            assert (float((want[row] - planted).abs().max()) < 0.05) == inside         # the case shows what it is meant to show
    K.check_device_errors()


# ------------------------------------------------------------------------------ the engine
LENS = [37, 100, 64, 19, 85, 50, 1, 2, 3, 160]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("tigelorn"))
    out = {}
    for name in ("T1", "T2", "T3"):
        d = TT.make_model_dir(name, root)
        cfg, w = TT.load_model_dir(d)
        reqs = {f"r{i}": tiny.random_tokens(cfg["vocab"], n, 100 + i) for i, n in enumerate(LENS)}
        out[name] = (d, cfg, w, reqs, {r: P.forward(cfg, w, t).float() for r, t in reqs.items()})
    return out


def _runner(model_dir, name, dtype, pool):
    from infurnace_b200.engine.loading import EngineOptions, build_runner
    ps = TT.TINY[name]["page_size"]
    return build_runner(model_dir, EngineOptions(dtype=dtype, device="cuda", page_size=ps, num_pages=pool // ps, max_num_seqs=4,
                                                 max_num_batched_tokens=pool, max_model_len=pool))[2]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", ["whole", "bulk_tail", "portions", "mixed"])
@pytest.mark.parametrize("name", ["T1", "T2", "T3"])
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


def test_the_fast_routes_ran(models):
    """The wider model's bfloat16 steps take the tensor-core attention kernels (bounded scores on tcgen05) and the chunked delta rule and scan; its layers
    would otherwise pass on the plain kernels alone."""
    d, cfg, w, reqs, ref = models["T3"]
    runner = _runner(d, "T3", "bfloat16", 640)
    k = runner.rt.kernels
    before = (k.latent_mma_calls, k.delta_chunked_calls, k.linear_scan_blocked_calls, k.stream_attention_calls, k.tc_attention_calls)
    tiny.run_inprocess(runner, tiny.schedule_whole({"a": reqs["r9"]}))
    assert k.latent_mma_calls > before[0] and k.delta_chunked_calls > before[1] and k.linear_scan_blocked_calls > before[2]
    assert k.stream_attention_calls == before[3] and k.tc_attention_calls > before[4]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_and_each_request_alone(models, dtype):
    """Unequal requests in one step against each alone: the same logits up to rounding."""
    d, cfg, w, reqs, ref = models["T3"]
    four = {r: reqs[r] for r in ("r9", "r6", "r3", "r1")}
    step = [{"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in four.items()], "end": list(four)}]
    runner = _runner(d, "T3", dtype, 640)
    together = tiny.collect(step, tiny.run_inprocess(runner, step), cfg["vocab"])
    for r, t in four.items():
        alone = tiny.collect(s := tiny.schedule_whole({r: t}), tiny.run_inprocess(runner, s), cfg["vocab"])[r]
        top = max(1.0, float(ref[r].abs().max()))
        close(together[r], alone, (2e-5 if dtype == "float32" else 0.06) * top, r)


OTHER_SIZES = {
    # widths that are no multiple of 8 (the plain products), heads of 24 + 10, ranks of 40 and 9, seven taps
    "odd": TT._config(53, 100, 1e-5, [
        TT._lat(3, 24, 10, 20, 40, 9, 0.2, 777.0, TT._dense(36)), TT._delta(3, 3, 20, 15, 7, 5, TT._dense(20)),
        TT._par((6, 2, 20, 12, 0.8, 3, 40.0, 6), (9, 7, (0.8, 0.9, 0.97)), (0.6, 1.4), None)], (97, 41, 2)),
    # sizes the tensor-core routes take throughout: heads of 128 and 64, ranks of 128 and 256, a window that is a page's
    # multiple, sixteen query heads per key head
    "tc": TT._config(211, 128, 1e-6, [
        _p := TT._par((16, 1, 128, 128, 0.06, 64, 5000.0, 64), (64, 128, (0.9, 0.97)), (1.0, 1.0), TT._dense(256)),
        TT._lat(16, 32, 16, 32, 128, 64, 0.15, 5000.0, TT._dense(128)), _c := TT._delta(2, 1, 128, 128, 4, 16),
        TT._lat(4, 64, 64, 64, 256, 128, 0.1, 20.0, None, scaling=None), TT._again([_p, None, _c], 2),
        TT._par((4, 2, 64, 128, 0.1, 50, 5000.0, 32), (128, 64, (0.99, 0.5)), (1.2, 0.3), None)], (1009, 3, 1)),
    # single layers
    "one": TT._config(40, 32, 1e-5, [TT._delta(2, 2, 16, 8, 2, 4, TT._dense(16))], (3, 1, 2)),
    "side": TT._config(40, 32, 1e-5, [TT._par((1, 1, 32, 16, 0.3, 10, 100.0, 32), (1, 1, (0.9,)), (1.0, 1.0), None)], (3, 1, 2)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(OTHER_SIZES))
def test_other_sizes_and_orders(tmp_path, name, dtype):
    """Models of other sizes, head counts and orders of layers, in a mixed schedule over a small pool."""
    from infurnace_b200.engine.loading import EngineOptions, build_runner
    conf = OTHER_SIZES[name]
    d = TT.make_model_dir("_" + name, str(tmp_path), config=conf, seed=31, store="bfloat16", sharpen=2.0)
    cfg, w = TT.load_model_dir(d)
    reqs = {f"r{i}": tiny.random_tokens(cfg["vocab"], n, 7 + i) for i, n in enumerate([45, 130, 3, 70, 1, 99, 20])}
    ref = {r: P.forward(cfg, w, t).float() for r, t in reqs.items()}
    steps = tiny.schedule_mixed(reqs, max_live=4, max_tokens=384, seed=3, sizes=(2, 3, 16, 21, 40, 64))
    runner = build_runner(d, EngineOptions(dtype=dtype, device="cuda", page_size=16, num_pages=24, max_num_seqs=4,
                                           max_num_batched_tokens=384, max_model_len=384))[2]
    out = tiny.collect(steps, tiny.run_inprocess(runner, steps), cfg["vocab"])
    runner.rt.kernels.check_device_errors()
    assert runner.cache.num_free_slots == 4 and runner.cache.free_pages() == [g.pool.num_pages for g in runner.cache.kv_groups]
    if dtype == "float32":
        for rid in reqs:
            rows_match(out[rid], ref[rid], dtype, f"{name} request {rid}")
    else:
        rows_match(torch.cat([out[r] for r in reqs]), torch.cat([ref[r] for r in reqs]), dtype, name, share=0.8)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_and_long_decoding(models, dtype):
    """Every token alone from the first on, 300 of them: windows of 33 and 120 pass over decoded tokens, pages of the windowed
    layers go back and come again, the recurrences run 300 steps from their slots."""
    d, cfg, w, _, _ = models["T3"]
    toks = tiny.random_tokens(cfg["vocab"], 300, 77)
    want = P.forward(cfg, w, toks).float()
    steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    out = tiny.collect(steps, tiny.run_inprocess(_runner(d, "T3", dtype, 384), steps), cfg["vocab"])["x"]
    rows_match(out, want, dtype, "token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_in_portions_then_decoding(models, dtype):
    """600 tokens: portions of 300, 133, 2 and 100, then 65 tokens one by one, beside a second request that comes and goes."""
    d, cfg, w, _, _ = models["T3"]
    toks = tiny.random_tokens(cfg["vocab"], 600, 91)
    other = tiny.random_tokens(cfg["vocab"], 90, 92)
    want, want_other = P.forward(cfg, w, toks).float(), P.forward(cfg, w, other).float()
    steps, at = [], 0
    for i, n in enumerate([300, 133, 2, 100] + [1] * 65):
        entries = [{"id": "x", "tokens": toks[at:at + n], "want": list(range(n))}]
        if i == 1:
            entries.append({"id": "y", "tokens": other[:60], "want": list(range(60))})
        if 2 <= i < 32:
            entries.append({"id": "y", "tokens": [other[58 + i]], "want": [0]})
        steps.append({"step": i, "entries": entries, "end": ["y"] if i == 31 else []})
        at += n
    assert at == 600
    out = tiny.collect(steps, tiny.run_inprocess(_runner(d, "T3", dtype, 768), steps), cfg["vocab"])
    rows_match(out["x"], want, dtype, "the long request")
    rows_match(out["y"], want_other, dtype, "the request beside it")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(models, tmp_path, dtype):
    d, cfg, w, reqs, ref = models["T2"]
    steps = tiny.schedule_mixed(reqs, max_live=4, max_tokens=640, seed=5)
    outputs = tiny.run_trace_run(d, dtype, steps, str(tmp_path / "out"), 640, TT.TINY["T2"]["page_size"])
    out = tiny.collect(steps, outputs, cfg["vocab"])
    rows_match(torch.cat([out[rid] for rid in reqs]), torch.cat([ref[rid] for rid in reqs]), dtype, "all requests")


def test_greedy_generation_through_the_engine_and_its_graphs(models):
    """The engine's own entry point: scheduler, portions beside decoded tokens, six requests over four slots, decode
    steps replayed from CUDA graphs (the token before is on the device only).  In float32 the tokens are the plain
    implementation's."""
    from infurnace_b200.engine import Engine, EngineOptions, SamplingParams
    d, cfg, w, _, _ = models["T1"]
    ps = TT.TINY["T1"]["page_size"]
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


def test_command_line(models, tmp_path):
    import json
    import os
    import subprocess
    import sys
    d, cfg, w, _, _ = models["T1"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "infurnace-b200"), "--model", d, "--prompt-ids", "5,6,7,8",
                          "--max-tokens", "6", "--json", "--dtype", "float32", "--page-size", "16", "--max-context", "64"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["generated_token_ids"] == P.greedy(cfg, w, [5, 6, 7, 8], 6) and report["model"]["architecture"] == "Tigelorn"
