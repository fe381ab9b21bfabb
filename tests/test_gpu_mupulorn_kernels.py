"""The kernels behind Mupulorn, each against the plain implementation: residual step with norms and convolution, PolyNorm,
capped logits, latent norms with rotation and scatter, per-head products, absorbed and expanded attention."""
import pytest
import torch

from oracle import mupulorn as P
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


def padded(t, width):
    out = torch.zeros(*t.shape[:-1], width, dtype=t.dtype)
    out[..., :t.shape[-1]] = t
    return out


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------ residual, norms, convolution
def run_sandwich(dtype, dim, taps, lens, new, per_channel=False, decode=False, run=0, embed=False, seed=0):
    """Sequences of lens tokens of which the last `new` are computed in this call; earlier tokens are in the state."""
    from nanovllm_b200 import ops
    dp, eps, B = pad8(dim), 1e-4, len(lens)
    table = rnd(seed + 90, 50, dim).to(dtype)
    ids = [torch.randint(0, 50, (n,), generator=torch.Generator().manual_seed(seed + b)) for b, n in enumerate(lens)]
    x = [(table[i].float() if embed else rnd(seed + 10 + b, n, dim)) for b, (i, n) in enumerate(zip(ids, lens))]
    y = [rnd(seed + 30 + b, n, dim).to(dtype) for b, n in enumerate(lens)]
    post, norm = (rnd(seed + 1, dim) + 1, rnd(seed + 2, dim) + 1) if per_channel else (torch.tensor([0.7]), torch.tensor([1.3]))
    w = (0.6 * rnd(seed + 3, dim, taps)).to(dtype) if taps else None
    slots = [2 * (B - b) - 1 for b in range(B)]
    state = torch.full((2 * B + 1, max(taps - 1, 0), dp), 5.0).to(dtype)  # leftovers of earlier sequences
    want_x, want_out, want_state = [], [], []
    for b in range(B):
        xb = x[b].double() if embed else x[b].double() + P.gain_norm(y[b].double(), post.double(), eps)
        h = P.gain_norm(xb, norm.double(), eps)
        if dtype == torch.bfloat16:
            h = h.float().bfloat16().double()  # what is kept, and convolved, is the rounded value
        out = h + P.causal_conv(h, w.double()) if taps else h
        k = lens[b] - new[b]
        want_x.append(xb[k:])
        want_out.append(out[k:])
        if taps > 1:
            z = torch.cat((torch.zeros(taps - 1, dim, dtype=torch.float64), h))
            want_state.append(z[len(z) - (taps - 1):])
            if k:
                state[slots[b]] = padded(z[k:k + taps - 1].to(dtype), dp)
    cat = lambda parts, d: padded(torch.cat([p[-m:] for p, m in zip(parts, new)]), d).to(DEV)
    padw = (lambda t: padded(t, dp) if t.numel() > 1 else t)
    cu = None if decode else i32([0] + torch.tensor(new).cumsum(0).tolist())
    cw = padded(w.T.contiguous(), dp).to(DEV) if taps else None
    sd = state.to(DEV)
    before = sd.clone()
    xd = None if embed else cat(x, dp)
    kw = dict(embed=(torch.cat([i[-m:] for i, m in zip(ids, new)]).to(DEV), padded(table, dp).to(DEV))) if embed else {}
    new_x, out = ops.sandwich_step(xd, None if embed else cat(y, dp), None if embed else padw(post).to(DEV), padw(norm).to(DEV), eps, dim,
                                   (cu, i32(lens), i32(slots), max(new)), cw, sd if taps else None, run=run, **kw)
    assert new_x[:, dim:].abs().sum() == 0 and out[:, dim:].abs().sum() == 0
    close(new_x[:, :dim], torch.cat(want_x), torch.float32, "residual")
    close(out[:, :dim], torch.cat(want_out), dtype, "output", 2)
    if taps > 1:
        for b in range(B):
            close(sd[slots[b], :, :dim], want_state[b], dtype, f"state of sequence {b}")
        rest = [i for i in range(state.shape[0]) if i not in slots]
        assert torch.equal(sd[rest], before[rest])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,taps", [(40, 1), (61, 2), (264, 3), (1024, 4), (72, 5), (2050, 9), (4100, 4), (4096, 4), (9000, 2), (96, 0)])
def test_residual_step(dtype, dim, taps):
    run_sandwich(dtype, dim, taps, [1, 2, 3, 7, 40], [1, 2, 3, 7, 40])
    run_sandwich(dtype, dim, taps, [5, 40, 9, 21], [2, 17, 1, 4], per_channel=True, seed=3)
    run_sandwich(dtype, dim, taps, [1, 2, 3, 30], [1, 1, 1, 1], decode=True, seed=4)


@pytest.mark.parametrize("run", [4, 5, 16])
def test_residual_step_across_the_runs_of_a_prompt(run):
    """Prompts cut into many runs, of which a run's first tokens are computed again; ends just at and around a run's edge."""
    for taps in (2, 4, 5):
        run_sandwich(torch.float32, 48, taps, [3 * run, 3 * run + 1, 3 * run - 1, run, run + 1, 200], [3 * run, 3 * run + 1, 3 * run - 1, run, run + 1, 200], run=run)
        run_sandwich(torch.bfloat16, 48, taps, [100, 3 * run + 20, 60], [90, 3 * run, run + 1], run=run, seed=7)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_starts_from_the_embedding(dtype):
    run_sandwich(dtype, 60, 3, [1, 20, 6], [1, 20, 2], embed=True)
    run_sandwich(dtype, 64, 4, [1, 5], [1, 1], embed=True, decode=True)


def test_padded_decode_rows_leave_every_state_alone():
    from nanovllm_b200 import ops
    state = torch.ones(2, 3, 16, device=DEV)
    x, y = torch.randn(3, 16, device=DEV), torch.randn(3, 16, device=DEV)
    one = torch.ones(1, device=DEV)
    _, out = ops.sandwich_step(x, y, one, one, 1e-5, 16, (None, i32([0, 4, 0]), i32([-1, 1, -1]), 1), torch.ones(4, 16, device=DEV), state)
    assert torch.isfinite(out).all() and (state[0] == 1).all() and not (state[1] == 1).all()


def test_last_step_does_not_store_the_residual():
    from nanovllm_b200 import ops
    x, y, one = torch.randn(5, 24, device=DEV), torch.randn(5, 24, device=DEV), torch.ones(1, device=DEV)
    before = x.clone()
    new_x, out = ops.sandwich_step(x, y, one, one, 1e-5, 24, (None, None, None, 1), store=False)
    want = P.gain_norm(x.double().cpu() + P.gain_norm(y.double().cpu(), 1.0, 1e-5), 1.0, 1e-5)
    assert new_x is None and torch.equal(x, before)
    close(out, want, torch.float32, "final norm")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim", [(3, 40), (301, 261), (2, 6001), (300, 18432), (5, 17000)])
def test_poly_norm(dtype, rows, dim):
    from nanovllm_b200 import ops
    z = (3 * rnd(1, rows, dim)).to(dtype)
    z[0, 0] = 40.0  # an outlier moves the root mean squares of the powers apart
    for coef in ([0.5, 0.25, 2.0, 0.1], [1.0, 0.0, 0.0, 0.0], [0.0, -1.0, 0.0, 0.0], [0.0, 0.0, 1.0, -3.0]):
        c = torch.tensor(coef)
        got = ops.poly_norm(padded(z, pad8(dim)).to(DEV), c.to(DEV), 1e-4, dim)
        close(got[:, :dim], P.poly_norm(z.double(), c.double(), 1e-4), dtype, f"{coef}")
        assert got[:, dim:].abs().sum() == 0
    small = (1e-3 * rnd(2, 4, dim)).to(dtype)  # the epsilon inside the root counts
    close(ops.poly_norm(padded(small, pad8(dim)).to(DEV), torch.ones(4, device=DEV), 1e-4, dim)[:, :dim], P.poly_norm(small.double(), torch.ones(4).double(), 1e-4), dtype, "small")


@pytest.mark.parametrize("dtype", DTYPES)
def test_capped_logits(dtype):
    from nanovllm_b200 import ops
    x = (40 * rnd(1, 5, 1304)).to(dtype)
    close(ops.logit_cap(x.to(DEV), 0.3, 7.0), P.capped(x.double(), 0.3, 7.0), torch.float32, "scaled and capped")
    close(ops.logit_cap(x.to(DEV), 0.3, 0.0), x.double() * 0.3, torch.float32, "scaled")


def test_sampling_uses_the_capped_logits():
    """One token far ahead of the rest, but the cap flattens it: the fused sampler must draw the others about as often as the
    capped distribution says."""
    from nanovllm_b200 import runtime as rt
    from nanovllm_b200.layers.embed_head import PaddedLMHead
    if rt.get_runtime().vocab != 1024:
        pytest.skip("another runtime is alive")
    torch.set_default_device(DEV)
    torch.set_default_dtype(torch.bfloat16)
    try:
        head = PaddedLMHead(1024, 64, scale=0.5, cap=2.0)
    finally:
        torch.set_default_device("cpu")
        torch.set_default_dtype(torch.float32)
    w = torch.zeros(1024, 64)
    w[:, 0] = -40.0
    w[:8, 0] = torch.tensor([30.0, 6.0, 4.0, 2.0, 0.0, -2.0, -4.0, -6.0])
    head.weight.data.copy_(w)
    x = torch.zeros(64, 64, device=DEV, dtype=torch.bfloat16)
    x[:, 0] = 1.0
    assert (head.head_sample(x, None, 11).cpu() == 0).all()
    hits = torch.zeros(1024, dtype=torch.float64)
    for _ in range(150):
        hits += torch.bincount(head.head_sample(x, torch.full((64,), 0.5, device=DEV), 11).cpu(), minlength=1024).double()
    p = torch.softmax(P.capped(w[:, 0].double(), 0.5, 2.0) / 0.5, -1)
    n = hits.sum()
    for i in range(8):
        assert abs(hits[i] - n * p[i]) < 5 * (n * p[i] * (1 - p[i])).sqrt() + 3, f"token {i}: {hits[i]} of {n}, expected {n * p[i]:.0f}"


# ------------------------------------------------------------------------------------------------ latents and the cache
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q,kv,rot", [(44, 52, 12), (80, 264, 64), (16, 8, 2), (300, 512, 34)])
def test_latent_norms_rotation_and_scatter(dtype, q, kv, rot):
    from nanovllm_b200 import ops
    from nanovllm_b200.layers.rotary_embedding import PairRotation
    M, eps, base = 9, 1e-4, 90.0
    qp, lp, rp = pad8(q), pad8(kv), pad8(rot)
    rope = PairRotation(rot, rot, base)
    rope.bind(3000, DEV)
    raw = [rnd(i, M, n).to(dtype) for i, n in enumerate((q, kv, rot))]
    rows = torch.cat([padded(t, pad8(t.shape[1])) for t in raw] + [torch.full((M, 8), 3.0, dtype=dtype)], 1).to(DEV)
    qw, kw = rnd(5, q) + 1, rnd(6, kv) + 1
    pos = torch.tensor([0, 1, 2, 63, 64, 700, 2999, 5, 1500])
    slots = [5, 0, 11, -1, 3, 7, 2, 9, 10]
    cache = torch.full((2, 6, 1, lp + rp), 7.0, dtype=dtype, device=DEV)
    ops.latent_store(rows, q, qp, kv, lp, rp, padded(qw, qp).to(DEV), padded(kw, lp).to(DEV), eps, pos.to(DEV), rope.table, cache, i32(slots))
    wq, wk = P.gain_norm(raw[0].double(), qw.double(), eps), P.gain_norm(raw[1].double(), kw.double(), eps)
    wr = P.rotate_pairs(raw[2].double(), pos, rot, base)
    close(rows[:, :q], wq, dtype, "query latent")
    close(rows[:, qp:qp + kv], wk, dtype, "latent")
    close(rows[:, qp + lp:qp + lp + rot], wr, dtype, "rotated part")
    assert (rows[:, qp + lp + rp:] == 3).all()
    flat = cache.view(12, lp + rp)
    for i, s in enumerate(slots):
        if s >= 0:
            assert torch.equal(flat[s], rows[i, qp:qp + lp + rp])
    for s in set(range(12)) - set(slots):
        assert (flat[s] == 7).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_gather_of_cached_rows(dtype):
    from nanovllm_b200 import ops
    cache = rnd(0, 9, 16, 1, 72).to(dtype).to(DEV)
    tables, lens = i32([[3, 8, 0], [5, 1, -1], [7, -1, -1]]), [40, 17, 1]
    cu = i32([0, 40, 57, 58])
    got = ops.latent_gather(cache, tables, cu, 40, 58)
    want = torch.cat([cache[tables[b, :-(-n // 16)].long()].reshape(-1, 72)[:n] for b, n in enumerate(lens)])
    assert torch.equal(got, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 24, 40), (64, 5, 136, 128), (65, 2, 64, 64), (200, 7, 520, 32), (3, 1, 8, 264)])
def test_one_product_per_head(dtype, M, H, N, K):
    from nanovllm_b200 import ops
    from nanovllm_b200.layers.rotary_embedding import PairRotation
    rot, rp, base = 12, 16, 90.0
    rope = PairRotation(rot, rot, base)
    rope.bind(500, DEV)
    x = rnd(0, M, H, K + rp).to(dtype)
    x[..., K + rot:] = 0
    pos = torch.randint(0, 500, (M,), generator=torch.Generator().manual_seed(1))
    w = (rnd(2, H, N + 16, K) / K ** 0.5).to(dtype)  # the rows of another matrix lie behind a head's
    want = torch.einsum("mhk,hnk->mhn", x[..., :K].double(), w[:, :N].double())
    got = ops.heads_gemm(x.view(M, -1).to(DEV), K + rp, w.to(DEV)[:, :N], False, N + rp, rotate=(rp, pos.to(DEV), rope.table)).view(M, H, N + rp)
    close(got[..., :N], want, dtype, "outputs by rows")
    close(got[..., N:N + rot], P.rotate_pairs(x[..., K:K + rot].double(), pos, rot, base), dtype, "rotated part")
    wt = w[:, :N].transpose(1, 2).contiguous()
    g = rnd(3, M, H * N + 8).to(dtype)
    got = ops.heads_gemm(x.view(M, -1).to(DEV), K + rp, wt.to(DEV), True, N, gate=g.to(DEV)[:, :H * N], gate_head=N).view(M, H, N)
    close(got, want * torch.sigmoid(g[:, :H * N].double()).view(M, H, N), dtype, "inputs by rows, gated", 1.5)


# ------------------------------------------------------------------------------------------------------------- attention
def plant(lat, q_lat, first_pos, strength, scale, heads):
    """For a few queries, one cached latent gets the query itself, scaled to score `strength`: the first key, the query's own
    position, the one before and the one AFTER it, keys at tile and page borders, far away and near."""
    spots = set()
    for t in sorted({0, len(q_lat) // 2, len(q_lat) - 1}):
        i = first_pos + t
        for j in (i + 1, i, i - 1, 0, 15, 16, 63, 64, 127, 128, i // 2):
            if 0 <= j < lat.shape[0] and j not in spots:
                h = len(spots) % heads
                qv = q_lat[t, h].float()
                lat[j] = (qv * strength / (scale * (qv @ qv))).to(lat.dtype)
                spots.add(j)


def run_latent(dtype, heads, L, rot, lens, q_lens, block=16, form=0, seed=0, decode=False, scale=0.11):
    from nanovllm_b200 import ops
    lp, rp = pad8(L), pad8(rot)
    g = torch.Generator().manual_seed(seed)
    lat, kr = [[torch.randn(n, w, generator=g).to(dtype) for n in lens] for w in (L, rot)]
    qn, qr = [[torch.randn(n, heads, w, generator=g).to(dtype) for n in q_lens] for w in (L, rot)]
    for b in range(len(lens)):
        plant(lat[b], qn[b], lens[b] - q_lens[b], 9.0, scale, heads)
    width = max(-(-n // block) for n in lens)
    perm = torch.randperm(len(lens) * width + 2, generator=g).tolist()
    tables = torch.full((len(lens), width), -1, dtype=torch.int32)
    cache = torch.randn(len(perm), block, 1, lp + rp, generator=g).to(dtype)
    for b, n in enumerate(lens):
        for t in range(-(-n // block)):
            tables[b, t] = perm.pop()
        for j in range(n):
            cache[int(tables[b, j // block]), j % block, 0] = torch.cat((padded(lat[b][j], lp), padded(kr[b][j], rp)))
    sink = 2 + 2 * torch.randn(heads, generator=g)
    M = sum(q_lens)
    q = torch.cat((padded(torch.cat(qn), lp), padded(torch.cat(qr), rp)), -1).reshape(M, -1)
    cu = None if decode else i32([0] + torch.tensor(q_lens).cumsum(0).tolist())
    got = ops.latent_attention(q.to(DEV), heads, cache.to(DEV), lp, tables.to(DEV), cu, i32(lens), max(q_lens), max(lens), scale, sink.to(DEV), form=form)
    at = 0
    for b, n in enumerate(q_lens):
        k = lat[b].double().unsqueeze(1).expand(-1, heads, -1)
        want = P.attend(qn[b].double(), qr[b].double(), k, kr[b].double(), k, scale, sink.double(), lens[b] - n)
        close(got[at:at + n].view(n, heads, lp)[..., :L], want, dtype, f"sequence {b}", 1.0 if dtype == torch.bfloat16 else 2.0)
        assert got[at:at + n].view(n, heads, lp)[..., L:].abs().sum() == 0
        at += n


# heads, latent, rotated part, block (a multiple of 128: tcgen05)
LATENT = [(5, 52, 12, 128), (16, 128, 64, 128), (20, 200, 34, 256), (33, 512, 64, 128), (1, 24, 2, 16), (40, 264, 40, 256), (7, 72, 8, 24), (32, 448, 64, 128)]
FORMS = [(torch.float32, 0), (torch.bfloat16, 0), (torch.bfloat16, 1)]


@pytest.mark.parametrize("case", range(len(LATENT)))
@pytest.mark.parametrize("dtype,form", FORMS)
def test_absorbed_attention_decode(case, dtype, form):
    heads, L, rot, block = LATENT[case]
    run_latent(dtype, heads, L, rot, [1, 2, 63, 64, 65, 128, 200, 300], [1] * 8, block, form, seed=case, decode=True)


@pytest.mark.parametrize("case", range(len(LATENT)))
@pytest.mark.parametrize("dtype,form", FORMS)
def test_absorbed_attention_prompts_and_portions(case, dtype, form):
    heads, L, rot, block = LATENT[case]
    run_latent(dtype, heads, L, rot, [1, 30, 70, 129, 66], [1, 30, 11, 2, 3], block, form, seed=case)


def test_absorbed_attention_split_over_many_ctas():
    """Long sequences whose key tiles go to many CTAs; repeated calls find their counters reset; a batch with a short one."""
    for rep in range(3):
        run_latent(torch.bfloat16, 6, 256, 32, [1500 + 37 * rep], [1], 128, seed=rep, decode=True)
    run_latent(torch.bfloat16, 18, 136, 64, [900, 5], [1, 1], 256, decode=True)
    run_latent(torch.bfloat16, 3, 512, 64, [700], [5], 128)
    run_latent(torch.bfloat16, 2, 64, 8, [9000], [1], 128, decode=True)


def test_absorbed_attention_when_the_running_maximum_keeps_rising():
    """Scores that grow from tile to tile by more and by less than the amount after which outputs are rescaled."""
    from nanovllm_b200 import ops
    heads, L, rot, n, scale = 5, 128, 8, 900, 0.1
    q = rnd(0, 1, heads, L + rot).bfloat16()
    for rise in (0.004, 0.05, 0.3):
        ramp = torch.arange(1024).view(8, 128, 1, 1) * rise
        unit = q[0].float().mean(0) / q[0].float().mean(0).pow(2).sum()
        c = (0.3 * rnd(1, 8, 128, 1, L + rot) + ramp * unit).bfloat16()
        kn = c.view(1024, L + rot)[:n, :L].double().unsqueeze(1).expand(-1, heads, -1)
        want = P.attend(q[:, :, :L].double(), q[:, :, L:].double(), kn, c.view(1024, L + rot)[:n, L:].double(), kn, scale, torch.zeros(heads).double(), n - 1)
        got = ops.latent_attention(q.view(1, -1).to(DEV), heads, c.to(DEV), L, torch.arange(8, dtype=torch.int32, device=DEV).view(1, 8), None, i32([n]), 1, 1024,
                                   scale, torch.zeros(heads, device=DEV))
        close(got.view(1, heads, L), want, torch.bfloat16, f"rise {rise}")


def test_absorbed_attention_of_wide_latents_runs_on_the_general_kernel():
    run_latent(torch.bfloat16, 2, 600, 72, [90], [9])
    run_latent(torch.float32, 2, 600, 72, [90, 40], [1, 1], decode=True)


def test_padded_decode_rows_give_zeros():
    from nanovllm_b200 import ops
    for dtype in DTYPES:
        cache = torch.randn(2, 128, 1, 80, device=DEV).to(dtype)
        out = ops.latent_attention(torch.randn(3, 160, device=DEV).to(dtype), 2, cache, 64, torch.zeros(3, 1, dtype=torch.int32, device=DEV), None,
                                   i32([4, 0, 0]), 1, 128, 0.1, torch.zeros(2, device=DEV))
        assert out[0].abs().sum() > 0 and out[1:].abs().sum() == 0


def run_expanded(heads, d, rot, dv, lens, q_lens, seed=0, scale=0.12, gated=True, base=300.0):
    from nanovllm_b200 import ops
    from nanovllm_b200.layers.rotary_embedding import PairRotation
    dtype, dp, rp, vp = torch.bfloat16, pad8(d), pad8(rot), pad8(dv)
    g = torch.Generator().manual_seed(seed)
    rope = PairRotation(rot, rot, base)
    rope.bind(max(lens), DEV)
    mk = lambda ns, *w: [torch.randn(n, *w, generator=g).to(dtype) for n in ns]
    kn, kr, v, qn, qr = mk(lens, heads, d), mk(lens, rot), mk(lens, heads, dv), mk(q_lens, heads, d), mk(q_lens, heads, rot)
    for b in range(len(lens)):
        for h in range(heads):
            plant(kn[b][:, h], qn[b][:, h:h + 1], lens[b] - q_lens[b], 9.0, scale, 1)
    sink = 2 + 2 * torch.randn(heads, generator=g)
    M, cat = sum(q_lens), torch.cat
    q = cat((padded(cat(qn), dp), padded(cat(qr), rp)), -1).reshape(M, -1)
    kv = cat((padded(cat(kn), dp), padded(cat(v), vp)), -1).reshape(sum(lens), -1)
    gate = torch.randn(M, heads, dv, generator=g).to(dtype)
    cu = lambda ns: i32([0] + torch.tensor(ns).cumsum(0).tolist())
    got = ops.expanded_attention(q.to(DEV), heads, kv.to(DEV), padded(cat(kr), rp + 8).to(DEV)[:, :rp], cu(q_lens), cu(lens), max(q_lens), dp, rp, vp, scale,
                                 sink.to(DEV), rope.table, padded(gate, vp).reshape(M, -1).to(DEV) if gated else None).view(M, heads, vp)
    at = 0
    for b, n in enumerate(q_lens):
        pos = torch.arange(lens[b] - n, lens[b])
        rotated = P.rotate_pairs(qr[b].double(), pos, rot, base).float().bfloat16().double()
        want = P.attend(qn[b].double(), rotated, kn[b].double(), kr[b].double(), v[b].double(), scale, sink.double(), lens[b] - n)
        if gated:
            want = want * torch.sigmoid(gate[at:at + n].double())
        close(got[at:at + n, :, :dv], want, dtype, f"sequence {b}")
        assert got[at:at + n, :, dv:].abs().sum() == 0
        at += n


@pytest.mark.parametrize("heads,d,rot,dv", [(3, 20, 12, 28), (2, 40, 20, 72), (4, 64, 64, 64), (2, 128, 64, 128), (1, 72, 2, 16), (2, 120, 40, 100), (5, 8, 8, 8)])
def test_expanded_attention(heads, d, rot, dv):
    run_expanded(heads, d, rot, dv, [1, 70, 150, 129, 66], [1, 70, 21, 1, 2])
    run_expanded(heads, d, rot, dv, [130, 64, 65], [130, 64, 63], seed=1, gated=False)
    run_expanded(heads, d, rot, dv, [300, 257, 40], [300, 130, 40], seed=2)


def test_expanded_attention_over_many_tiles():
    """Longer sequences: every slot of the rings is used again, both query tiles and one of them alone, a late short portion."""
    run_expanded(2, 128, 64, 128, [900, 1100, 513], [900, 600, 129], seed=3)
    run_expanded(1, 64, 32, 64, [1500, 700], [300, 3], seed=4)
    run_expanded(3, 72, 8, 104, [640, 641], [640, 257], seed=5, scale=0.4)  # sharp scores: outputs are rescaled on the way
