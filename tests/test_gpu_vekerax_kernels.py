"""The kernels behind Vekerax, each against the plain implementation: residual streams, head norm and scatter, window
attention, decayed linear attention, gated norm, fp32 and activated matrix products."""
import pytest
import torch

from oracle import vekerax as V
from tests.gpu_util import ensure_group

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 1.5e-2}  # relative to the row's largest value; bf16: a few roundings of 2^-9


@pytest.fixture(scope="module", autouse=True)
def runtime(pkg):
    ensure_group()
    from nanovllm_b200 import runtime as rt
    created = rt._RUNTIME is None
    if created:
        rt.init_runtime(max_tokens=2048, hidden=1024, oneshot_tokens=256, vocab=1024, max_seqs=64)
    yield
    if created:
        rt.shutdown_runtime()


def rnd(seed, *shape):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def close(got, want, dtype, what, factor=1.0):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    bound = TOL[dtype] * factor * want.abs().amax(-1, keepdim=True).clamp_min(1e-3)
    err = (got - want).abs()
    assert (err <= bound).all(), f"{what}: {(err / bound).max().item():.2f} of the bound at {torch.nonzero(err > bound)[:4].tolist()}"


def pad8(n):
    return (n + 7) // 8 * 8


# ---------------------------------------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams,dim,rows", [(1, 40, 3), (2, 61, 5), (3, 264, 301), (4, 1024, 2), (4, 2050, 300), (5, 72, 7), (8, 4100, 4), (9, 96, 3), (4, 4099, 3), (2, 9000, 2)])
def test_stream_step(dtype, streams, dim, rows):
    from nanovllm_b200 import ops
    dp, eps, m = pad8(dim), 1e-4, 0.37
    x, y = rnd(1, rows, streams, dim), rnd(2, rows, dim).to(dtype)
    mix, w_out, w_in, nw = rnd(3, streams, streams), rnd(4, streams), rnd(5, streams), rnd(6, dim)
    xp = torch.zeros(rows, streams, dp)
    xp[..., :dim] = x
    yp = torch.zeros(rows, dp, dtype=dtype)
    yp[:, :dim] = y
    nwp = torch.zeros(dp)
    nwp[:dim] = nw
    xd = xp.to(DEV)
    got = ops.stream_step(xd, yp.to(DEV), mix.to(DEV), w_out.to(DEV), m, w_in.to(DEV), nwp.to(DEV), eps, dim)
    want_x = V.stream_update(x.double(), y.double(), mix.double(), w_out.double(), m)
    want = V.rms_norm(V.stream_input(want_x, w_in.double()), nw.double(), eps)
    close(xd[..., :dim].reshape(rows, -1), want_x.reshape(rows, -1), torch.float32, "streams")
    close(got[:, :dim], want, dtype, "normed")
    assert got[:, dim:].abs().sum() == 0 and xd[..., dim:].abs().sum() == 0
    before = xd.clone()
    last = ops.stream_step(xd, yp.to(DEV), mix.to(DEV), w_out.to(DEV), m, None, nwp.to(DEV), eps, dim, store=False)
    want = V.rms_norm(V.stream_update(want_x, y.double(), mix.double(), w_out.double(), m).sum(1), nw.double(), eps)
    close(last[:, :dim], want, dtype, "sum of the streams", 2)
    assert torch.equal(before, xd)


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_start_from_the_embedding(dtype):
    from nanovllm_b200 import ops
    table, ids, nw, w_in = rnd(1, 50, 96).to(dtype), torch.tensor([3, 49, 0, 3]), rnd(2, 96), rnd(3, 3)
    x = torch.empty(4, 3, 96, device=DEV)
    got = ops.stream_step(x, None, None, None, 0.0, w_in.to(DEV), nw.to(DEV), 1e-5, 96, embed=(ids.to(DEV), table.to(DEV), 1.7))
    e = V.embedding(ids.tolist(), table.double(), 1.7)
    close(x.reshape(4, -1), e.unsqueeze(1).repeat(1, 3, 1).reshape(4, -1), torch.float32, "streams")
    close(got, V.rms_norm(e * w_in.double().sum(), nw.double(), 1e-5), dtype, "normed", 2)


# --------------------------------------------------------------------------------------------------- matrix products
@pytest.mark.parametrize("M", [1, 5, 64, 100, 300, 700])
def test_activated_products_match_the_equations(M):
    from nanovllm_b200 import _abi, ops
    for dtype in DTYPES:
        x, w = rnd(1, M, 136).to(dtype), (rnd(2, 336, 136) / 12).to(dtype)
        y = x.double() @ w.double().T
        want = torch.cat((V.silu(y[:, :200]), y[:, 200:]), 1)
        close(ops.gemm(x.to(DEV), w.to(DEV), silu_cols=200), want, dtype, f"silu columns {dtype}")
        got = ops.gemm_act_mul(x.to(DEV), w.to(DEV), _abi.ACT_RELU)
        close(got, torch.relu(y[:, 0::2]) * y[:, 1::2], dtype, f"relu pairs {dtype}", 2)
        close(ops.gemm_act_mul(x.to(DEV), w.to(DEV), _abi.ACT_SILU), V.silu(y[:, 0::2]) * y[:, 1::2], dtype, f"silu pairs {dtype}", 2)


# ------------------------------------------------------------------------------------------------- head norm, scatter
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,d,dv", [(4, 2, 24, 40), (3, 3, 33, 7), (6, 1, 128, 64), (2, 1, 264, 16)])
def test_head_norm_and_scatter(dtype, nq, nkv, d, dv):
    from nanovllm_b200 import ops
    M, eps, dp, vp = 9, 1e-4, pad8(d), pad8(dv)
    qkv = torch.zeros(M, nq * dp + nkv * (dp + vp), dtype=dtype)
    raw = rnd(1, M, nq + nkv, d).to(dtype)
    v = rnd(2, M, nkv, dv).to(dtype)
    qkv[:, :(nq + nkv) * dp].view(M, nq + nkv, dp)[..., :d] = raw
    qkv[:, (nq + nkv) * dp:].view(M, nkv, vp)[..., :dv] = v
    qw, kw = torch.zeros(dp, dtype=dtype), torch.zeros(dp, dtype=dtype)
    qw[:d], kw[:d] = rnd(3, d).to(dtype), rnd(4, d).to(dtype)
    slots = torch.tensor([5, 0, 11, -1, 3, 7, 2, 9, 10], dtype=torch.int32)
    kc, vc = torch.full((2, 6, nkv, dp), 7.0, dtype=dtype, device=DEV), torch.full((2, 6, nkv, vp), 7.0, dtype=dtype, device=DEV)
    qd = qkv.to(DEV)
    ops.qk_norm_store(qd, nq, nkv, d, dp, dv, vp, qw.to(DEV), kw.to(DEV), eps, kc, vc, slots.to(DEV))
    wq = V.rms_norm(raw[:, :nq].double(), qw[:d].double(), eps)
    wk = V.rms_norm(raw[:, nq:].double(), kw[:d].double(), eps)
    close(qd[:, :nq * dp].view(M, nq, dp)[..., :d], wq, dtype, "q")
    kf, vf = kc.view(12, nkv, dp), vc.view(12, nkv, vp)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kf[s, :, :d], wk[i], dtype, "k")
            assert torch.equal(vf[s, :, :dv].cpu(), v[i])
    for s in {1, 4, 6, 8} & set(range(12)):
        assert (kf[s] == 7).all() and (vf[s] == 7).all()


@pytest.mark.parametrize("M", [3, 64, 200])
def test_projection_with_head_norm_in_the_epilogue(M):
    """128-wide heads without rotation: one launch up to 64 tokens, two above; the same values either way."""
    from nanovllm_b200 import ops
    nq, nkv, K, eps = 3, 2, 256, 1e-5
    x, w = rnd(1, M, K).bfloat16(), (rnd(2, (nq + 2 * nkv) * 128, K) / 16).bfloat16()
    qw, kw = rnd(3, 128).bfloat16(), rnd(4, 128).bfloat16()
    kc, vc = torch.zeros(2, 128, nkv, 128, dtype=torch.bfloat16, device=DEV), torch.zeros(2, 128, nkv, 128, dtype=torch.bfloat16, device=DEV)
    slots = torch.randperm(256, generator=torch.Generator().manual_seed(0))[:M].int()
    got = ops.qkv_fused(x.to(DEV), w.to(DEV), None, nq, nkv, 128, qw.to(DEV), kw.to(DEV), eps, None, None, kc, vc, slots.to(DEV))
    y = (x.double() @ w.double().T).view(M, nq + 2 * nkv, 128)
    close(got.view(M, -1, 128)[:, :nq], V.rms_norm(y[:, :nq], qw.double(), eps), torch.bfloat16, "q")
    close(kc.view(256, nkv, 128)[slots.long().to(DEV)], V.rms_norm(y[:, nq:nq + nkv], kw.double(), eps), torch.bfloat16, "k")
    close(vc.view(256, nkv, 128)[slots.long().to(DEV)], y[:, nq + nkv:], torch.bfloat16, "v")


# -------------------------------------------------------------------------------------------------- window attention
class Paged:
    """Sequences of random K/V in a paged cache with shuffled blocks; query i's needles are keys that score far above the
    rest just inside and just outside the window and among the first tokens, so that a wrong edge changes the output."""

    def __init__(self, dtype, lens, nkv, d, dv, block, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.d, self.dv, self.dp, self.vp = d, dv, pad8(d), pad8(dv)
        width = max(-(-n // block) for n in lens)
        perm = torch.randperm(len(lens) * width + 3, generator=g).tolist()
        self.k = [torch.randn(n, nkv, d, generator=g).to(dtype) for n in lens]
        self.v = [torch.randn(n, nkv, dv, generator=g).to(dtype) for n in lens]
        self.tables = torch.zeros(len(lens), width, dtype=torch.int32)
        self.kc = torch.randn(len(perm), block, nkv, self.dp, generator=g).to(dtype)
        self.vc = torch.randn(len(perm), block, nkv, self.vp, generator=g).to(dtype)
        self.kc[..., d:] = 0
        self.vc[..., dv:] = 0
        self.block, self.lens, self.dtype = block, lens, dtype
        for b, n in enumerate(lens):
            for t in range(-(-n // block)):
                self.tables[b, t] = perm.pop()
        self.write()

    def write(self):
        for b, n in enumerate(self.lens):
            for j in range(n):
                at = (int(self.tables[b, j // self.block]), j % self.block)
                self.kc[at][:, :self.d] = self.k[b][j]
                self.vc[at][:, :self.dv] = self.v[b][j]


def plant(p, b, q, first_pos, window, keep, scale, strength=9.0):
    """For a few query rows, one key near an edge gets q itself (scaled to score `strength`)."""
    tq, heads, _ = q.shape
    nkv = p.k[b].shape[1]
    spots = []
    for t in sorted({0, tq // 3, tq // 2, tq - 1}):
        i = first_pos + t
        for j in (i - window, i - window + 1, keep - 1, keep, i, i - 1):
            if 0 <= j < p.lens[b] and all(abs(j - s) > 0 for s in spots) and len(spots) < tq + 6:
                g = len(spots) % nkv
                qv = q[t, g * (heads // nkv)].float()
                p.k[b][j, g] = (qv * strength / (scale * (qv @ qv))).to(p.dtype)
                p.v[b][j, g] = (p.v[b][j, g].float() + 3.0).to(p.dtype)
                spots.append(j)


def run_attention(dtype, lens, q_lens, heads, nkv, d, dv, scale, cap, window, keep, with_sink, block=16, form=0, seed=0, decode=False):
    from nanovllm_b200 import ops
    p = Paged(dtype, lens, nkv, d, dv, block, seed)
    q = [rnd(seed + 50 + b, n, heads, d).to(dtype) for b, n in enumerate(q_lens)]
    for b in range(len(lens)):
        plant(p, b, q[b], lens[b] - q_lens[b], window, keep, scale)
    p.write()
    sink = rnd(seed + 9, heads) if with_sink else None
    M = sum(q_lens)
    qp = torch.zeros(M, heads * p.dp + 8, dtype=dtype)  # a row longer than the heads, as in a merged projection
    qp[:, :heads * p.dp].view(M, heads, p.dp)[..., :d] = torch.cat(q)
    cu = torch.tensor([0] + torch.tensor(q_lens).cumsum(0).tolist(), dtype=torch.int32)
    got = ops.window_attention(qp.to(DEV), heads, p.kc.to(DEV), p.vc.to(DEV), p.tables.to(DEV), None if decode else cu.to(DEV),
                               torch.tensor(lens, dtype=torch.int32, device=DEV), max(q_lens), max(lens), scale, cap, window, keep,
                               sink.to(DEV) if with_sink else None, form=form)
    got = got.view(M, heads, p.vp)
    at = 0
    for b, n in enumerate(q_lens):
        want = V.attention_core(q[b].double(), p.k[b].double(), p.v[b].double(), scale, cap if cap > 0 else 1e9, window, keep,
                                sink.double() if with_sink else torch.full((heads,), -1e30, dtype=torch.float64), lens[b] - n)
        # bf16: the output's own rounding; fp32: exponentials and sums
        close(got[at:at + n, :, :dv], want, dtype, f"sequence {b}", 1.0 if dtype == torch.bfloat16 else 2.0)
        assert got[at:at + n, :, dv:].abs().sum() == 0
        at += n


ATTN = [  # heads, kv_heads, dim, vdim, scale, cap, window, keep, sink, block
    (4, 1, 24, 40, 0.2, 20.0, 7, 2, True, 16),
    (6, 2, 64, 64, 0.1, 50.0, 64, 4, True, 32),
    (8, 8, 128, 128, 0.09, 30.0, 65, 0, False, 16),
    (3, 1, 80, 48, 0.15, 0.0, 1, 1, True, 24),
    (5, 5, 128, 72, 0.09, 5.0, 100, 70, True, 64),
    (20, 1, 40, 128, 0.2, 20.0, 33, 63, True, 8),
    (4, 2, 56, 56, 0.2, 20.0, 10 ** 9, 0, True, 256),
]


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("dtype,form", [(torch.float32, 0), (torch.bfloat16, 0), (torch.bfloat16, 1)])
def test_window_attention_prefill(case, dtype, form):
    heads, nkv, d, dv, scale, cap, window, keep, sink, block = ATTN[case]
    # whole prompts, the first tokens, a portion after a cached prefix that ends at block and window edges, two tokens
    run_attention(dtype, [1, 70, 150, 129, 66], [1, 70, 21, 1, 2], heads, nkv, d, dv, scale, cap, window, keep, sink, block, form, seed=case)


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("dtype,form", [(torch.float32, 0), (torch.bfloat16, 0), (torch.bfloat16, 1)])
def test_window_attention_decode(case, dtype, form):
    heads, nkv, d, dv, scale, cap, window, keep, sink, block = ATTN[case]
    run_attention(dtype, [1, 2, 63, 64, 65, 128, 200, 700], [1] * 8, heads, nkv, d, dv, scale, cap, window, keep, sink, block, form, seed=case, decode=True)


def test_window_attention_decode_split_over_many_ctas():
    """One long sequence: its key tiles go to many CTAs whose parts are combined; repeated calls find their counters reset."""
    for rep in range(3):
        run_attention(torch.bfloat16, [3000 + 37 * rep], [1], 4, 2, 128, 128, 0.09, 30.0, 2500, 5, True, 64, seed=rep, decode=True)
    run_attention(torch.bfloat16, [900, 5], [1, 1], 4, 2, 64, 128, 0.1, 30.0, 10 ** 6, 0, True, 64, decode=True)


def test_window_attention_wide_heads_run_on_the_general_kernel():
    run_attention(torch.bfloat16, [90], [90], 2, 1, 200, 264, 0.07, 30.0, 20, 3, True)
    run_attention(torch.float32, [90, 40], [1, 1], 2, 1, 200, 264, 0.07, 30.0, 20, 3, True, decode=True)


def test_padded_decode_rows_give_zeros():
    from nanovllm_b200 import ops
    for dtype in DTYPES:
        kc = torch.randn(2, 16, 1, 64, device=DEV).to(dtype)
        out = ops.window_attention(torch.randn(3, 128, device=DEV).to(dtype), 2, kc, kc, torch.zeros(3, 1, dtype=torch.int32, device=DEV), None,
                                   torch.tensor([4, 0, 0], dtype=torch.int32, device=DEV), 1, 16, 0.1, 20.0, 8, 2, torch.zeros(2, device=DEV))
        assert out[0].abs().sum() > 0 and out[1:].abs().sum() == 0


# -------------------------------------------------------------------------------------------------- linear attention
def run_linear(dtype, heads, d, dv, decay, lens, new, form=0, seed=0, decode=False, slots=None):
    """Sequences of lens tokens of which the last `new` are computed in this call, from the state of the rest."""
    from nanovllm_b200 import ops
    dp, vp, B = pad8(d), pad8(dv), len(lens)
    g = torch.Generator().manual_seed(seed)
    mk = lambda n, w: (torch.randn(n, heads, w, generator=g) * (w ** -0.25)).to(dtype)
    q, k, v = ([mk(n, w) for n in lens] for w in (d, d, dv))
    slots = slots or list(reversed(range(B)))
    state = torch.full((max(slots) + 2, heads, dp, vp), 5.0)  # leftovers of earlier sequences
    rows, want_o, want_s = [], [], []
    for b, (n, m) in enumerate(zip(lens, new)):
        _, s0 = V.lightning_core(q[b][:n - m].double(), k[b][:n - m].double(), v[b][:n - m].double(), decay) if n > m else (None, None)
        o, s = V.lightning_core(q[b][n - m:].double(), k[b][n - m:].double(), v[b][n - m:].double(), decay, s0)
        if s0 is not None:
            state[slots[b]] = 0
            state[slots[b], :, :d, :dv] = s0.float()
        want_o.append(o)
        want_s.append(s)
        r = torch.zeros(m, heads * (2 * dp + vp) + 8, dtype=dtype)
        r[:, :heads * dp].view(m, heads, dp)[..., :d] = q[b][n - m:]
        r[:, heads * dp:2 * heads * dp].view(m, heads, dp)[..., :d] = k[b][n - m:]
        r[:, 2 * heads * dp:heads * (2 * dp + vp)].view(m, heads, vp)[..., :dv] = v[b][n - m:]
        rows.append(r)
    dec = torch.tensor(decay, dtype=torch.float64)
    powers = (dec.unsqueeze(1) ** torch.arange(65)).float()
    cu = torch.tensor([0] + torch.tensor(new).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
    sd = state.to(DEV)
    o = ops.linear_attn(torch.cat(rows).to(DEV), heads, dp, vp, sd, torch.tensor(slots, dtype=torch.int32, device=DEV), None if decode else cu,
                        torch.tensor(lens, dtype=torch.int32, device=DEV), max(new), dec.float().to(DEV), powers.to(DEV), form=form)
    at = 0
    for b, m in enumerate(new):
        # products of exact bf16 inputs with a 16-bit split of the fp32 factors: far below one bf16 rounding
        close(o[at:at + m].view(m, heads, vp)[..., :dv], want_o[b], torch.float32, f"output of sequence {b}", 4)
        close(sd[slots[b], :, :d, :dv].reshape(heads, -1), want_s[b].reshape(heads, -1), torch.float32, f"state of sequence {b}", 1 if dtype == torch.float32 else 4)
        at += m
    untouched = [i for i in range(state.shape[0]) if i not in slots]
    assert torch.equal(sd[untouched].cpu(), state[untouched])


LIN = [(3, 20, 28, [0.6, 0.9, 0.999]), (2, 64, 64, [0.99, 1.0]), (2, 128, 128, [0.3, 0.995]), (1, 72, 136, [0.97]), (2, 128, 40, [0.0, 0.9])]


@pytest.mark.parametrize("case", range(len(LIN)))
@pytest.mark.parametrize("dtype,form", [(torch.float32, 0), (torch.bfloat16, 0), (torch.bfloat16, 1)])
def test_linear_attention_prompts_and_portions(case, dtype, form):
    heads, d, dv, decay = LIN[case]
    run_linear(dtype, heads, d, dv, decay, [1, 2, 63, 64, 65, 130], [1, 2, 63, 64, 65, 130], form, seed=case)
    run_linear(dtype, heads, d, dv, decay, [40, 66, 200, 129], [1, 2, 70, 65], form, seed=case + 10, slots=[3, 7, 0, 4])


@pytest.mark.parametrize("case", [1, 2, 3])
def test_linear_attention_across_segments(case):
    """Prompts long enough to be cut into segments that run side by side, next to short ones, fresh and continued."""
    heads, d, dv, decay = LIN[case]
    run_linear(torch.bfloat16, heads, d, dv, decay, [511, 512, 513, 1100, 3], [511, 512, 513, 1100, 3], seed=case)
    run_linear(torch.bfloat16, heads, d, dv, decay, [700, 1090, 5], [600, 1025, 2], seed=case + 5, slots=[2, 0, 5])


def test_linear_attention_many_heads_walk_long_prompts_in_one_piece():
    run_linear(torch.bfloat16, 130, 16, 24, [0.5 + i / 270 for i in range(130)], [600, 585], [600, 520])


@pytest.mark.parametrize("case", range(len(LIN)))
@pytest.mark.parametrize("dtype,form", [(torch.float32, 0), (torch.bfloat16, 0), (torch.bfloat16, 1)])
def test_linear_attention_decode(case, dtype, form):
    heads, d, dv, decay = LIN[case]
    run_linear(dtype, heads, d, dv, decay, [1, 2, 50, 9], [1, 1, 1, 1], form, seed=case, decode=True, slots=[1, 6, 0, 3])


def test_linear_attention_wide_heads_run_on_the_general_kernel():
    run_linear(torch.bfloat16, 2, 200, 48, [0.9, 0.99], [70, 20], [70, 5])


def test_linear_attention_padded_decode_rows():
    from nanovllm_b200 import ops
    for dtype in DTYPES:
        state = torch.ones(2, 1, 16, 16, device=DEV)
        o = ops.linear_attn(torch.randn(2, 48, device=DEV).to(dtype), 1, 16, 16, state, torch.tensor([-1, 1], dtype=torch.int32, device=DEV), None,
                            torch.tensor([0, 4], dtype=torch.int32, device=DEV), 1, torch.tensor([0.9], device=DEV),
                            (0.9 ** torch.arange(65, device=DEV)).view(1, 65).contiguous())
        assert o[0].abs().sum() == 0 and o[1].abs().sum() > 0 and (state[0] == 1).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim", [(3, 40), (300, 264), (2, 6000), (5, 17000)])
def test_gated_norm(dtype, rows, dim):
    from nanovllm_b200 import ops
    o, gate, w = rnd(1, rows, dim), rnd(2, rows, dim).to(dtype), rnd(3, dim)
    got = ops.gated_norm(o.to(DEV), gate.to(DEV), w.to(DEV), 1e-4, dim)
    close(got, V.gated_norm(o.double(), gate.double(), w.double(), 1e-4), dtype, "gated norm")
