"""The Gebelorn design on the GPU: every kernel of latent attention and of the fp32 stream, the model in fp32 and bf16
through the engine (captured decode steps included), against the plain statement in ``gebelorn_oracle``."""
import pytest
import torch

import gebelorn_cases as cases
import gebelorn_oracle as oracle
from pisceslx_b200.models.latent_attention import rotary_for
from pisceslx_b200.ops import latent as L

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _dev(t, dtype=None):
    return t.to("cuda", dtype) if dtype is not None else t.cuda()


def _rnd(g, *s):
    return torch.randn(*s, generator=g).bfloat16().float()          # values both dtypes hold exactly


def _close(got, want, dtype, scale=1.0):
    tol = (2e-2 if dtype == torch.bfloat16 else 2e-5) * scale
    err = (got.float().cpu() - want.float()).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), err


def _status_clean():
    from pisceslx_b200.ops import check_status
    torch.cuda.synchronize()
    check_status()


# ---- stream, activations, products ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [1, 50, 256, 1028, 2048, 4096, 8192, 8196])
def test_stream_norm(cols, dtype):
    g = torch.Generator().manual_seed(cols)
    T, eps = 5, 1e-3
    x, y, w1, w2 = torch.randn(T, cols, generator=g), _rnd(g, T, cols), _rnd(g, cols), _rnd(g, cols)
    table, ids = _rnd(g, 9, cols), torch.tensor([8, 0, 3, 3, 7])
    xs = _dev(x)
    h = L.stream_norm(xs, _dev(y, dtype), _dev(w1, dtype), _dev(w2, dtype), eps, dtype)
    want = x + oracle.rms(y, w1, eps)
    _close(xs, want, torch.float32)
    _close(h, oracle.rms(want, w2, eps), dtype)
    h = L.stream_norm(xs, _dev(y, dtype), _dev(w1, dtype), None, eps, dtype)
    _close(h, want + oracle.rms(y, w1, eps), dtype)
    h = L.stream_norm(xs, None, None, _dev(w2, dtype), eps, dtype)
    _close(h, oracle.rms(want + oracle.rms(y, w1, eps), w2, eps), dtype)
    h = L.stream_norm(xs, _dev(table, dtype), _dev(w1, dtype), _dev(w2, dtype), eps, dtype, rows=_dev(ids), start=True)
    want = oracle.rms(table[ids], w1, eps)
    _close(xs, want, torch.float32)
    _close(h, oracle.rms(want, w2, eps), dtype)
    _status_clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [3, 24, 64])
def test_gelu_and_token_gate(dim, dtype):
    g = torch.Generator().manual_seed(dim)
    z = 3 * _rnd(g, 7, dim + 5)
    _close(L.gelu(_dev(z, dtype)), oracle.gelu_erf(z), dtype)
    a, table, ids = 2 * _rnd(g, 7, dim), _rnd(g, 11, 4 * dim), torch.tensor([0, 10, 5, 5, 1, 2, 9])
    got = L.token_gate(_dev(a, dtype), _dev(table, dtype), 2 * dim, _dev(ids))
    _close(got, oracle.gelu_tanh(a) * table[ids][:, 2 * dim:3 * dim], dtype)
    _status_clean()


def test_index_outside_a_table_is_reported_not_read():
    from pisceslx_b200.ops import KernelStatusError, check_status
    table = torch.ones(4, 8, device="cuda", dtype=torch.bfloat16)
    out = L.token_gate(torch.ones(2, 8, device="cuda", dtype=torch.bfloat16), table, 0, torch.tensor([1, 4], device="cuda"))
    with pytest.raises(KernelStatusError):
        torch.cuda.synchronize()
        check_status()
    assert out[1].abs().max() == 0 and out[0].abs().min() > 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 8, 24), (3, 61, 50), (130, 104, 80), (70, 520, 264), (257, 7, 13)])
def test_project(M, N, K, dtype):
    g = torch.Generator().manual_seed(M + N + K)
    x, w = _rnd(g, M, K), _rnd(g, N, K)
    _close(L.project(_dev(x, dtype), _dev(w, dtype)), x @ w.T, dtype)
    _close(L.project(_dev(x, dtype), _dev(w, dtype), out_fp32=True), x @ w.T, torch.float32)
    _status_clean()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,B,N,K", [(3, 5, 40, 24), (2, 1, 256, 128), (5, 130, 136, 72), (2, 3, 9, 7)])
def test_project_heads_into_a_pitched_view(H, B, N, K, dtype):
    g = torch.Generator().manual_seed(H + B + N)
    R = L.head_rows(B, torch.empty(0, device="cuda", dtype=dtype))
    a, w = torch.zeros(H, R, K), _rnd(g, H, N, K)
    a[:, :B] = _rnd(g, H, B, K)
    out = torch.full((H, R, N + 8), 7.0, device="cuda", dtype=dtype)
    L.project_heads(_dev(a, dtype), _dev(w, dtype), out[:, :, :N], B)
    _close(out[:, :B, :N], torch.einsum("hmk,hnk->hmn", a[:, :B], w), dtype)
    assert (out[:, :, N:] == 7.0).all()                              # the columns next to the view are untouched
    _status_clean()


# ---- latent attention ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,rank,rot", [(13, 21, 6), (104, 144, 32), (64, 512, 64)])
def test_prep_norms_rotates_and_stores(q_rank, rank, rot, dtype):
    g = torch.Generator().manual_seed(rank)
    T, eps, row = 6, 1e-4, rank + rot
    y, wq, wk = _rnd(g, T, q_rank + row + 3), _rnd(g, q_rank), _rnd(g, rank)
    pos = torch.tensor([0, 1, 5, 63, 64, 700], dtype=torch.int32)
    spec = {"dims": rot, "base": 900.0, "yarn": cases.YARN}
    cos, sin = rotary_for(spec).tables(701, torch.device("cuda"))
    cache = torch.zeros(3, 4, row, device="cuda", dtype=dtype)
    slots = torch.tensor([11, -1, 0, 3, 5, 4], dtype=torch.int32, device="cuda")
    cq, rows = L.latent_prep(_dev(y, dtype), q_rank, rank, rot, _dev(wq, dtype), _dev(wk, dtype), cos, sin, _dev(pos), eps,
                             cache, slots)
    rotspec = {"dims": rot, "base": 900.0, "scaling": cases.YARN}
    want = torch.cat([oracle.rms(y[:, q_rank:q_rank + rank], wk, eps),
                      torch.stack([oracle.rotate(y[t, q_rank + rank:q_rank + row], int(pos[t]), rotspec) for t in range(T)])], 1)
    _close(cq, oracle.rms(y[:, :q_rank], wq, eps), dtype)
    _close(rows, want, dtype)
    flat = cache.view(-1, row)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], rows[t])
    assert flat[[1, 2, 6, 7, 8, 9, 10]].abs().max() == 0
    assert torch.equal(L.latent_gather(cache, slots[[0, 2, 5]]), rows[[0, 2, 5]])
    _status_clean()


def _prompt_case(g, lens, H, dim, rot, vdim):
    nq, nk = [a for a, _ in lens], [b for _, b in lens]
    Tq, Tk = sum(nq), sum(nk)
    q, k, v, kr = 1.5 * _rnd(g, Tq, H * (dim + rot)), 1.5 * _rnd(g, Tk, H * dim), _rnd(g, Tk, H * vdim), _rnd(g, Tk, rot)
    cu = lambda xs: torch.tensor([0] + torch.tensor(xs).cumsum(0).tolist(), dtype=torch.int32)
    return q, k, v, kr, cu(nq), cu(nk)


def _prompt_want(q, k, v, kr, gate, cq, ck, H, window, scale):
    out = []
    for b in range(len(cq) - 1):
        q0, q1, k0, k1 = int(cq[b]), int(cq[b + 1]), int(ck[b]), int(ck[b + 1])
        for i in range(q1 - q0):
            last = i + (k1 - k0) - (q1 - q0)
            js = oracle.visible(last, k1 - k0, window)
            lo, hi = k0 + js[0], k0 + js[-1] + 1
            qh = q[q0 + i].view(H, -1)
            dim = k.shape[1] // H
            o = oracle.attend(qh[:, :dim], qh[:, dim:], k[lo:hi].view(hi - lo, H, -1), kr[lo:hi], v[lo:hi].view(hi - lo, H, -1), scale)
            out.append((o * torch.sigmoid(gate[q0 + i])[:, None]).reshape(-1))
    return torch.stack(out)


@pytest.mark.parametrize("dtype,simt", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("H,dim,rot,vdim,window,lens", [
    (3, 64, 32, 48, 100, [(1, 1), (300, 300), (2, 131)]),
    (2, 128, 64, 128, 128, [(257, 400), (5, 5)]),
    (2, 24, 8, 40, 1, [(140, 140)]),
    (1, 72, 40, 72, None, [(130, 390), (64, 64)]),
    (2, 64, 16, 120, 129, [(128, 128), (129, 257)]),
])
def test_prompt_attention(H, dim, rot, vdim, window, lens, dtype, simt):
    g = torch.Generator().manual_seed(dim + rot)
    q, k, v, kr, cq, ck = _prompt_case(g, lens, H, dim, rot, vdim)
    gate = _rnd(g, q.shape[0], H)
    scale = (dim + rot) ** -0.5
    want = _prompt_want(q, k, v, kr, gate, cq, ck, H, window, scale)
    got = L.latent_attention(_dev(q, dtype), _dev(k, dtype), _dev(v, dtype), _dev(kr, dtype), _dev(gate, dtype), _dev(cq),
                             _dev(ck), max(a for a, _ in lens), H, window, scale, simt=simt)
    _status_clean()
    _close(got, want, dtype)


@pytest.mark.parametrize("simt", [False, True])
@pytest.mark.parametrize("window", [1, 2, 127, 128, 129])
@pytest.mark.parametrize("far", [0, 5, 127, 128])
def test_prompt_window_edge(window, far, simt):
    """One key takes all the weight of every query that sees it, and none of any other."""
    T, d, r = 300, 64, 32
    g = torch.Generator().manual_seed(far)
    q, k, v, kr = torch.zeros(T, d + r), 0.01 * _rnd(g, T, d), _rnd(g, T, d), 0.01 * _rnd(g, T, r)
    q[:, 0], k[far, 0] = 1.0, 60.0
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    bf = torch.bfloat16
    got = L.latent_attention(_dev(q, bf), _dev(k, bf), _dev(v, bf), _dev(kr, bf), None, cu, cu, T, 1, window, 1.0, simt=simt)
    _status_clean()
    hit = (got.float().cpu() - v[far]).abs().amax(1) < 0.05
    assert hit.tolist() == [far <= t < far + window for t in range(T)]


def _decode_case(g, lens, H, rank, rot, pages=40, block=64):
    row = rank + rot
    B = len(lens)
    width = max(-(-n // block) for n in lens) + 2
    cache = _rnd(g, pages, block, row)
    q = _rnd(g, H, B, row)
    table = torch.full((B, width), -1, dtype=torch.int32)
    perm = torch.randperm(pages, generator=g).tolist()
    for b, n in enumerate(lens):
        for i in range(-(-n // block)):
            table[b, i] = perm.pop()
    return cache, q, table


def _decode_want(cache, q, table, lens, rank, window, scale):
    H, B, row = q.shape
    bs = cache.shape[1]
    out = torch.zeros(H, B, rank)
    for b, n in enumerate(lens):
        js = torch.tensor(oracle.visible(n - 1, n, window))
        rows = cache[table[b].long()[js // bs], js % bs]
        w = torch.softmax((q[:, b] @ rows.T) * scale, -1)
        out[:, b] = w @ rows[:, :rank]
    return out


@pytest.mark.parametrize("dtype,simt", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("H,rank,rot,window,splits", [(5, 128, 40, 80, 1), (16, 512, 64, 300, 3), (20, 256, 64, None, 2),
                                                       (40, 512, 64, 128, 1), (70, 64, 8, 65, 2), (3, 136, 24, 1, 1),
                                                       (33, 200, 40, None, 7)])
def test_latent_decode(H, rank, rot, window, splits, dtype, simt):
    g = torch.Generator().manual_seed(H + rank)
    lens = [1, 63, 64, 65, 129, 400, 641]
    cache, q, table = _decode_case(g, lens, H, rank, rot)
    scale = 2.0 * (rank + rot) ** -0.5
    R = L.head_rows(len(lens), torch.empty(0, device="cuda", dtype=dtype))
    qp = torch.zeros(H, R, rank + rot)
    qp[:, :len(lens)] = q
    sl = torch.tensor(lens, dtype=torch.int32, device="cuda")
    if window:                                          # pages out of reach are placeholders: they must not be touched
        for b, n in enumerate(lens):
            table[b, :max(0, n - window) // 64] = -1
    got = L.latent_decode(_dev(qp, dtype), _dev(cache, dtype), rank, _dev(table), sl, window, scale, simt=simt, splits=splits)
    _status_clean()
    full = table.clone().clamp_min(0)
    _close(got[:, :len(lens)], _decode_want(cache, q, full, lens, rank, window, scale), dtype)


@pytest.mark.parametrize("simt", [False, True])
@pytest.mark.parametrize("window", [1, 63, 64, 65, 128])
def test_decode_window_edge(window, simt):
    """A step sees the standing-out key exactly while it is within the window, across page borders."""
    H, rank, rot = 2, 64, 16
    g = torch.Generator().manual_seed(window)
    far, bf = 70, torch.bfloat16
    lens = [71, 72, 70 + window, 71 + window, 132 + window]
    cache, q, table = _decode_case(g, lens, H, rank, rot, pages=64)
    cache, q = 0.01 * cache, torch.zeros_like(q)
    q[:, :, 0] = 1.0
    for b in range(len(lens)):
        cache[table[b, far // 64].long(), far % 64, 0] = 60.0
    R = L.head_rows(len(lens), torch.empty(0, device="cuda", dtype=bf))
    qp = torch.zeros(H, R, rank + rot)
    qp[:, :len(lens)] = q
    out = L.latent_decode(_dev(qp, bf), _dev(cache, bf), rank, _dev(table), torch.tensor(lens, dtype=torch.int32, device="cuda"),
                          window, 1.0, simt=simt)
    _status_clean()
    seen = (out[0, :len(lens), 0].float().cpu() > 50).tolist()
    assert seen == [n - 1 - far < window for n in lens]


def test_rescaled_sums_when_later_keys_score_far_higher():
    """Scores grow from page to page, so that the running maximum moves in every tile."""
    H, rank, rot, n = 5, 128, 32, 640
    g = torch.Generator().manual_seed(4)
    cache, q, table = _decode_case(g, [n], H, rank, rot)
    for i in range(n):
        cache[table[0, i // 64].long(), i % 64, 0] = 12.0 * (i // 64)
    q[:, :, 0] = 1.0
    bf = torch.bfloat16
    cache = cache.bfloat16().float()
    qp = torch.zeros(H, 128, rank + rot)
    qp[:, :1] = q
    for splits in (1, 4):
        got = L.latent_decode(_dev(qp, bf), _dev(cache, bf), rank, _dev(table), torch.tensor([n], dtype=torch.int32, device="cuda"),
                              None, 1.0, splits=splits)
        _status_clean()
        _close(got[:, :1], _decode_want(cache, q, table, [n], rank, None, 1.0), bf)


# ---- the model ------------------------------------------------------------------------------------------------------
EXACT = 3e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make", [cases.mixed, cases.odd, cases.wide])
def test_every_cut_gives_the_plain_logits(make, dtype):
    cfg = make()
    W = cases.weights(cfg, 1)
    m = cases.build(cfg, W, "cuda", dtype)
    toks = cases.tokens(cfg, 230)
    want = cases.expected(cfg, W, toks, torch.float32)
    limit = cases.rounding_limit(cfg, W, toks, want) if dtype == torch.bfloat16 else torch.full((len(toks),), EXACT)
    eng = cases.engine(m)
    for name, cuts in cases.CUTS.items():
        ratio = cases.error(cases.run_cut(eng, 0, toks, cuts), want) / limit
        assert ratio.max() < 1, (name, ratio.max().item(), ratio.argmax().item())
    assert eng.graph.disabled_reason is None and eng.graph.replays > 0
    _status_clean()


def test_pages_are_released_and_used_again_during_captured_decoding():
    cfg = cases.mixed()
    W = cases.weights(cfg, 2)
    m = cases.build(cfg, W, "cuda", torch.float32)
    eng = cases.engine(m, blocks=8)                      # 8 pages of 64 for 700 tokens; one is the padding page
    toks = cases.tokens(cfg, 700)
    want = cases.expected(cfg, W, toks, torch.float32)
    got = cases.run_cut(eng, 3, toks, [120, 90, 1])
    assert cases.error(got, want).max() < EXACT
    assert eng.cache.alloc.available() == 7


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_requests_equal_each_alone(dtype):
    """Unequal requests decode together through the scheduler; greedy tokens are the plain ones (fp32) and every
    request's tokens are those it gets alone."""
    cfg = cases.mixed()
    W = cases.weights(cfg, 7)
    m = cases.build(cfg, W, "cuda", dtype)
    prompts = [cases.tokens(cfg, n, seed=30 + n) for n in (1, 3, 64, 129, 40, 77)]
    new = [25, 40, 9, 30, 3, 70]
    eng = cases.engine(m, blocks=40)
    reqs = [eng.add_request(p, max_new_tokens=n) for p, n in zip(prompts, new)]
    eng.run_until_done()
    if dtype == torch.float32:
        for r, p in zip(reqs, prompts):
            seq = p + r.output_ids
            logits = cases.expected(cfg, W, seq, torch.float32)
            assert logits[len(p) - 1:-1].argmax(-1).tolist() == r.output_ids
    else:
        for r, p, n in zip(reqs, prompts, new):
            # teacher-forced alone: the batch's choice is within rounding of the best logit
            alone = cases.run_cut(eng, 100 + r.request_id, p + r.output_ids, [len(p), 1])
            pick = alone[len(p) - 1:-1].gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
            spread = alone.std()
            assert (alone[len(p) - 1:-1].amax(1) - pick).max() < 0.1 * spread
    _status_clean()
