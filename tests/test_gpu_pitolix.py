"""The Pitolix design on the GPU: every kernel of grouped attention over pages and of the parallel stream, the model in
fp32 and bf16 through the engine (captured decode steps included), against the plain statement in ``pitolix_oracle``."""
import pytest
import torch

import pitolix_cases as cases
import pitolix_oracle as oracle
from pisceslx_b200.models.latent_attention import rotary_for
from pisceslx_b200.ops import functional as F_
from pisceslx_b200.ops import grouped as G
from pisceslx_b200.ops import latent as L

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
PATHS = [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)]


def _dev(t, dtype=None):
    return None if t is None else t.to("cuda", dtype) if dtype is not None else t.cuda()


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


# ---- stream, activation, products ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [1, 50, 256, 1028, 2048, 4096, 8192, 8196])
def test_stream_add(cols, dtype):
    g = torch.Generator().manual_seed(cols)
    T, eps = 5, 1e-3
    x, parts = torch.randn(T, cols, generator=g), torch.randn(3, T + 3, cols, generator=g)
    w1, w2, vec, table, ids = _rnd(g, cols), _rnd(g, cols), _rnd(g, cols), _rnd(g, 9, cols), torch.tensor([8, 0, 3, 3, 7])
    xs = _dev(x)
    h1, h2 = L.stream_add(xs, _dev(parts), (_dev(w1, dtype), _dev(w2, dtype)), 1.0, eps, dtype, table=_dev(table, dtype),
                          rows=_dev(ids), table_scale=2.5, vec=_dev(vec, dtype))
    want = x + parts[:, :T].sum(0) + 2.5 * table[ids] + vec
    _close(xs, want, torch.float32)
    _close(h1, oracle.norm(want, w1, eps), dtype)
    _close(h2, oracle.norm(want, w2, eps), dtype)
    before = xs.clone()
    (h,) = L.stream_add(xs, None, (_dev(w2, dtype),), 0.0, eps, dtype)
    _close(h, oracle.unit(want, eps) * w2, dtype)
    assert torch.equal(xs, before)
    assert L.stream_add(xs, _dev(parts[0, :T].contiguous()), (), 0.0, eps, dtype) == ()
    _close(xs, want + parts[0, :T], torch.float32)
    (h,) = L.stream_add(xs, None, (_dev(w1, dtype),), 1.0, eps, dtype, table=_dev(table, dtype), rows=_dev(ids), start=True)
    _close(xs, table[ids], torch.float32)
    _close(h, oracle.norm(table[ids], w1, eps), dtype)
    _status_clean()


def test_a_token_outside_the_table_is_reported_not_read():
    from pisceslx_b200.ops import KernelStatusError, check_status
    x = torch.zeros(2, 8, device="cuda")
    L.stream_add(x, None, (), 0.0, 1e-6, torch.bfloat16, table=torch.ones(4, 8, device="cuda", dtype=torch.bfloat16),
                 rows=torch.tensor([1, 4], device="cuda"), start=True)
    with pytest.raises(KernelStatusError):
        torch.cuda.synchronize()
        check_status()
    assert x[0].min() == 1.0 and x[1].abs().max() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,col", [(3, 1), (24, 8), (1000, 16), (96, 5)])
def test_gated_silu_into_a_column_range(ff, col, dtype):
    g = torch.Generator().manual_seed(ff)
    z = 4 * _rnd(g, 7, 2 * ff)
    out = torch.full((7, ff + col + 4), 7.0, device="cuda", dtype=dtype)
    L.swiglu(_dev(z, dtype), out[:, col:col + ff])
    a = z[:, :ff]
    _close(out[:, col:col + ff], a * torch.sigmoid(a) * z[:, ff:], dtype)
    assert (out[:, :col] == 7.0).all() and (out[:, col + ff:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 8, 24), (3, 61, 50), (130, 104, 80), (70, 520, 1024), (300, 256, 512), (128, 64, 2048)])
def test_product_onto_the_stream(M, N, K, dtype):
    """Added by the product itself, or handed over in parts."""
    g = torch.Generator().manual_seed(M + N + K)
    x, z, w = torch.randn(M, N, generator=g), _rnd(g, M, K), _rnd(g, N, K)
    xs = _dev(x)
    parts = L.project_onto(xs, _dev(z, dtype), _dev(w, dtype))
    if dtype == torch.bfloat16 and M <= 128 and K >= 512:
        assert parts is not None and parts.dim() == 3 and F_.skinny_parts(_dev(z, dtype), _dev(w, dtype)) is not None
    if parts is not None:
        L.stream_add(xs, parts, (), 0.0, 1e-6, dtype)
    _close(xs, x + z @ w.T, torch.float32, scale=3.0)
    _status_clean()


# ---- prep ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,unit,temp,bias", [
    (9, 3, 64, 56, 48, False, None, True), (4, 4, 128, 128, 0, True, (0.3, 5), False), (5, 1, 24, 104, 16, True, (0.2, 1), True),
    (3, 3, 10, 9, 6, True, (0.4, 64), True), (2, 1, 200, 16, 128, True, None, False), (2, 2, 16, 8, 8, False, None, True),
    (8, 2, 128, 64, 128, True, (1.0, 7), True)])
def test_prep(heads, kv, dim, vdim, rot, unit, temp, bias, dtype):
    g = torch.Generator().manual_seed(dim + vdim)
    T, eps = 6, 1e-3
    nq, nk, nv = heads * dim, kv * dim, kv * vdim
    at = [0, -(-nq // 8) * 8, -(-nq // 8) * 8 + -(-nk // 8) * 8]
    y = _rnd(g, T, at[2] + -(-nv // 8) * 8 + 8)
    b = 0.5 * _rnd(g, y.shape[1]) if bias else None
    pos = torch.tensor([0, 1, 5, 63, 64, 700], dtype=torch.int32)
    temp = {"coef": temp[0], "every": temp[1]} if temp else None
    rotspec = {"dims": rot, "base": 900.0}
    cos = sin = None
    if rot:
        cos, sin = rotary_for(rotspec).tables(701, torch.device("cuda"))
    kp, vp = torch.zeros(3, 4, kv, dim, device="cuda", dtype=dtype), torch.zeros(3, 4, kv, vdim, device="cuda", dtype=dtype)
    slots = torch.tensor([11, -1, 0, 3, 5, 4], dtype=torch.int32)
    ys = _dev(y, dtype)
    q, k, v = ys[:, :nq], ys[:, at[1]:at[1] + nk], ys[:, at[2]:at[2] + nv]
    G.grouped_prep(q, k, v, _dev(b, dtype), at, heads, kv, kp, vp, _dev(slots), _dev(pos), cos, sin, rot, unit, temp, eps)
    _status_clean()
    full = y + b if bias else y
    wq, wk, wv = full[:, :nq].view(T, heads, dim), full[:, at[1]:at[1] + nk].view(T, kv, dim), full[:, at[2]:at[2] + nv]
    if unit:
        wq, wk = oracle.unit(wq, eps), oracle.unit(wk, eps)
    if rot:
        wq, wk = (torch.stack([oracle.rotate(t[i], int(pos[i]), rotspec) for i in range(T)]) for t in (wq, wk))
    if temp:
        wq = torch.stack([wq[i] * oracle.temperature(int(pos[i]), temp) for i in range(T)])
    _close(q, wq.reshape(T, nq), dtype)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            _close(kp.view(12, kv, dim)[s], wk[t], dtype)
            _close(vp.view(12, -1)[s], wv[t], dtype)
    assert kp.view(12, -1)[[1, 2, 6, 7, 8, 9, 10]].abs().max() == 0 and vp.view(12, -1)[[1, 2, 6, 7, 8, 9, 10]].abs().max() == 0
    rows = torch.zeros(T, 1, kv, dim, device="cuda", dtype=dtype), torch.zeros(T, 1, kv, vdim, device="cuda", dtype=dtype)
    ys = _dev(y, dtype)
    G.grouped_prep(ys[:, :nq], ys[:, at[1]:at[1] + nk], ys[:, at[2]:at[2] + nv], _dev(b, dtype), at, heads, kv, *rows, None,
                   _dev(pos), cos, sin, rot, unit, temp, eps)
    _close(rows[0].view(T, -1), wk.reshape(T, -1), dtype)
    _close(rows[1].view(T, -1), wv, dtype)


# ---- attention -------------------------------------------------------------------------------------------------------
def _paged(g, lens, kv, dim, vdim, block=64, pages=48):
    """Pages in random order; whatever they hold next to the sequences' tokens is not a number."""
    kp, vp = torch.full((pages, block, kv, dim), float("nan")), torch.full((pages, block, kv, vdim), float("nan"))
    table = torch.full((len(lens), max(-(-n // block) for n in lens) + 2), -1, dtype=torch.int32)
    perm, ks, vs = torch.randperm(pages, generator=g).tolist(), [], []
    for b, n in enumerate(lens):
        for i in range(-(-n // block)):
            table[b, i] = perm.pop()
        k, v = 1.5 * _rnd(g, n, kv, dim), _rnd(g, n, kv, vdim)
        at = table[b].long()[torch.arange(n) // block] * block + torch.arange(n) % block
        kp.view(-1, kv, dim)[at], vp.view(-1, kv, vdim)[at] = k, v
        ks.append(k)
        vs.append(v)
    return kp, vp, table, ks, vs


def _want(q, ks, vs, nq, heads, scale, sink, gate):
    """q [Tq, heads * dim] packed: the last nq[b] positions of sequence b."""
    out, at = [], 0
    for k, v, n in zip(ks, vs, nq):
        for i in range(n):
            last = k.shape[0] - n + i
            o = oracle.attend(q[at].view(heads, -1), k[:last + 1], v[:last + 1], scale, sink)
            if gate is not None:
                o = o * torch.sigmoid(gate[at]).view(heads, -1)
            out.append(o.reshape(-1))
            at += 1
    return torch.stack(out)


SHAPES = [  # heads, kv_heads, dim, vdim, sink, gate
    (6, 3, 64, 56, True, "element"), (8, 1, 128, 128, False, "head"), (3, 3, 24, 40, True, "head"), (6, 2, 72, 16, True, None),
    (20, 1, 48, 128, False, "element"), (5, 5, 16, 8, False, None), (34, 2, 128, 64, True, "element")]


@pytest.mark.parametrize("dtype,simt", PATHS)
@pytest.mark.parametrize("heads,kv,dim,vdim,with_sink,with_gate", SHAPES)
def test_prompt_portions_over_pages(heads, kv, dim, vdim, with_sink, with_gate, dtype, simt):
    g = torch.Generator().manual_seed(dim + vdim)
    cases_ = [(1, 1), (2, 131), (150, 150), (129, 300), (3, 64), (64, 192)]
    nq, lens = [a for a, _ in cases_], [b for _, b in cases_]
    kp, vp, table, ks, vs = _paged(g, lens, kv, dim, vdim)
    T, scale = sum(nq), 1.3 * dim ** -0.5
    q = _rnd(g, T, heads * dim)
    sink = 2 * _rnd(g, heads) if with_sink else None
    gate = 2 * _rnd(g, T, heads * (vdim if with_gate == "element" else 1)) if with_gate else None
    cu = torch.tensor([0] + torch.tensor(nq).cumsum(0).tolist(), dtype=torch.int32)
    out = torch.full((T, heads * vdim + 16), 7.0, device="cuda", dtype=dtype)
    G.grouped_attention(_dev(q, dtype), _dev(kp, dtype), _dev(vp, dtype), _dev(table), _dev(torch.tensor(lens, dtype=torch.int32)),
                        _dev(cu), max(nq), heads, scale, _dev(sink, dtype), _dev(gate, dtype), out[:, 8:8 + heads * vdim], simt=simt)
    _status_clean()
    _close(out[:, 8:8 + heads * vdim], _want(q, ks, vs, nq, heads, scale, sink, gate), dtype)
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + heads * vdim:] == 7.0).all()


@pytest.mark.parametrize("dtype,simt", PATHS)
@pytest.mark.parametrize("heads,kv,dim,vdim,with_sink,with_gate", SHAPES[:4])
def test_prompts_in_packed_rows(heads, kv, dim, vdim, with_sink, with_gate, dtype, simt):
    g = torch.Generator().manual_seed(dim)
    lens = [1, 130, 5, 64, 257]
    T, scale = sum(lens), dim ** -0.5
    q, k, v = _rnd(g, T, heads * dim), 1.5 * _rnd(g, T, kv, dim), _rnd(g, T, kv, vdim)
    sink = 2 * _rnd(g, heads) if with_sink else None
    cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32)
    out = torch.empty(T, heads * vdim, device="cuda", dtype=dtype)
    G.grouped_attention(_dev(q, dtype), _dev(k.unsqueeze(1), dtype), _dev(v.unsqueeze(1), dtype), None, None, _dev(cu), max(lens),
                        heads, scale, _dev(sink, dtype), None, out, simt=simt)
    _status_clean()
    _close(out, _want(q, k.split(lens), v.split(lens), lens, heads, scale, sink, None), dtype)


@pytest.mark.parametrize("dtype,simt", PATHS)
@pytest.mark.parametrize("splits", [1, 3, 7])
@pytest.mark.parametrize("heads,kv,dim,vdim,with_sink,with_gate", SHAPES)
def test_decode_over_pages(heads, kv, dim, vdim, with_sink, with_gate, splits, dtype, simt):
    g = torch.Generator().manual_seed(dim + vdim + splits)
    lens = [1, 63, 64, 65, 128, 129, 400, 641]
    B, scale = len(lens), 1.3 * dim ** -0.5
    kp, vp, table, ks, vs = _paged(g, lens, kv, dim, vdim)
    y = _rnd(g, B, heads * dim + 24)
    sink = 2 * _rnd(g, heads) if with_sink else None
    gate = 2 * _rnd(g, B, heads * (vdim if with_gate == "element" else 1)) if with_gate else None
    out = torch.full((B, heads * vdim + 16), 7.0, device="cuda", dtype=dtype)
    G.grouped_decode(_dev(y, dtype)[:, 8:8 + heads * dim], _dev(kp, dtype), _dev(vp, dtype), _dev(table),
                     _dev(torch.tensor(lens, dtype=torch.int32)), heads, scale, _dev(sink, dtype), _dev(gate, dtype),
                     out[:, 8:8 + heads * vdim], simt=simt, splits=splits)
    _status_clean()
    _close(out[:, 8:8 + heads * vdim], _want(y[:, 8:8 + heads * dim], ks, vs, [1] * B, heads, scale, sink, gate), dtype)
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + heads * vdim:] == 7.0).all()


@pytest.mark.parametrize("simt", [False, True])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 200])
def test_a_standing_out_key_is_seen_from_its_own_position_on(far, simt):
    """One key takes all the weight of every query at or behind it, and none of any other, in prompts and in decoding."""
    n, d, bf = 300, 64, torch.bfloat16
    g = torch.Generator().manual_seed(far)
    kp, vp, table, ks, vs = _paged(g, [n], 1, d, d)
    at = table[0].long()[torch.arange(n) // 64] * 64 + torch.arange(n) % 64
    kp.view(-1, d)[at] = 0.01 * ks[0].view(n, d)
    kp.view(-1, d)[at[far], 0] = 60.0
    q = torch.zeros(n, d)
    q[:, 0] = 1.0
    K, V, tab = _dev(kp, bf), _dev(vp, bf), _dev(table)
    v = vs[0].view(n, d)
    for m in (n, 2, 130):
        out = torch.empty(m, d, device="cuda", dtype=bf)
        G.grouped_attention(_dev(q[n - m:], bf), K, V, tab, torch.tensor([n], dtype=torch.int32, device="cuda"),
                            torch.tensor([0, m], dtype=torch.int32, device="cuda"), m, 1, 1.0, None, None, out, simt=simt)
        hit = (out.float().cpu() - v[far]).abs().amax(1) < 0.05
        assert hit.tolist() == [far <= t for t in range(n - m, n)]
    lens = [max(far, 1), far + 1, far + 2, n]
    out = torch.empty(4, d, device="cuda", dtype=bf)
    G.grouped_decode(_dev(q[:4], bf), K, V, tab.expand(4, -1).contiguous(), torch.tensor(lens, dtype=torch.int32, device="cuda"),
                     1, 1.0, None, None, out, simt=simt)
    _status_clean()
    hit = (out.float().cpu() - v[far]).abs().amax(1) < 0.05
    assert hit.tolist() == [far < m for m in lens]


@pytest.mark.parametrize("splits", [1, 4])
def test_rescaled_sums_when_later_keys_score_far_higher(splits):
    """Scores grow from page to page, so that the reference maximum moves in every tile; a sink of the middle height."""
    heads, d, n, bf = 5, 64, 640, torch.bfloat16
    g = torch.Generator().manual_seed(4)
    kp, vp, table, ks, vs = _paged(g, [n], 1, d, d)
    for i in range(n):
        ks[0][i, 0, 0] = 12.0 * (i // 64)
        kp[table[0, i // 64].long(), i % 64, 0, 0] = 12.0 * (i // 64)
    q = _rnd(g, 1, heads, d)
    q[:, :, 0] = 1.0
    q, sink = q.view(1, -1), torch.tensor([0.0, 60.0, 108.0, 112.0, 300.0])
    out = torch.empty(1, heads * d, device="cuda", dtype=bf)
    G.grouped_decode(_dev(q, bf), _dev(kp, bf), _dev(vp, bf), _dev(table), torch.tensor([n], dtype=torch.int32, device="cuda"),
                     heads, 1.0, _dev(sink, bf), None, out, splits=splits)
    want = _want(q, ks, vs, [1], heads, 1.0, sink, None)
    _close(out, want, bf)
    G.grouped_attention(_dev(q, bf), _dev(kp, bf), _dev(vp, bf), _dev(table), torch.tensor([n], dtype=torch.int32, device="cuda"),
                        torch.tensor([0, 1], dtype=torch.int32, device="cuda"), 1, heads, 1.0, _dev(sink, bf), None, out)
    _close(out, want, bf)
    _status_clean()


# ---- the model -------------------------------------------------------------------------------------------------------
EXACT = 3e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make", [cases.mixed, cases.odd, cases.wide, cases.plain])
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_after_every_run_of_a_layer(dtype):
    cfg = cases.mixed()
    W = cases.weights(cfg, 6)
    m, toks, ref, seen = cases.build(cfg, W, "cuda", dtype), cases.tokens(cfg, 150), [], []
    cases.expected(cfg, W, toks, torch.float32, layers_out=ref)
    for n in (150, 40):                                  # the product adds to the stream itself, or hands over parts
        seen.clear()
        m.model.layer_tap = lambda i, x: seen.append(x.float().cpu().clone())
        m(input_ids=torch.tensor([toks[:n]], device="cuda"))
        m.model.layer_tap = None
        for x, r in zip(seen, ref):
            assert (x - r[:n]).abs().max() < (3e-2 if dtype == torch.bfloat16 else 2e-5) * r.abs().max()
        assert len(seen) == len(ref) == 8


def test_long_captured_decoding_and_pages_used_again():
    cfg = cases.mixed()
    W = cases.weights(cfg, 2)
    m = cases.build(cfg, W, "cuda", torch.float32)
    eng = cases.engine(m, blocks=12)                     # one is the padding page; 600 tokens need ten
    toks = cases.tokens(cfg, 600)
    want = cases.expected(cfg, W, toks, torch.float32)
    assert cases.error(cases.run_cut(eng, 3, toks, [120, 90, 1]), want).max() < EXACT
    assert eng.cache.alloc.available() == 11
    for t in eng.cache.k + eng.cache.v:
        t.fill_(float("nan"))                            # whatever the pages still hold must not matter
    assert cases.error(cases.run_cut(eng, 4, toks[:200], [100, 2, 1]), want[:200]).max() < EXACT
    bf = cases.build(cfg, W, "cuda", torch.bfloat16)
    eng = cases.engine(bf, blocks=12)
    for t in eng.cache.k + eng.cache.v:
        t.fill_(float("nan"))
    limit = cases.rounding_limit(cfg, W, toks[:200], want[:200])
    for cuts in ([200], [100, 2, 1]):
        assert (cases.error(cases.run_cut(eng, 4, toks[:200], cuts), want[:200]) / limit).max() < 1
    _status_clean()


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
    for r, p, n in zip(reqs, prompts, new):
        assert len(r.output_ids) == n
        if dtype == torch.float32:
            logits = cases.expected(cfg, W, p + r.output_ids, torch.float32)
            assert logits[len(p) - 1:-1].argmax(-1).tolist() == r.output_ids
        else:
            # teacher-forced alone: the batch's choice is within rounding of the best logit
            alone = cases.run_cut(eng, 100 + r.request_id, p + r.output_ids, [len(p), 1])
            pick = alone[len(p) - 1:-1].gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
            assert (alone[len(p) - 1:-1].amax(1) - pick).max() < 0.1 * alone.std()
    _status_clean()


def test_generate_entry_point():
    cfg = cases.plain()
    W = cases.weights(cfg, 8)
    m = cases.build(cfg, W, "cuda", torch.float32)
    ids = torch.tensor([cases.tokens(cfg, 70, seed=1), cases.tokens(cfg, 70, seed=2)], device="cuda")
    out, _ = m.generate(ids, max_new_tokens=8)
    for row in out.tolist():
        assert row[70:] == cases.expected(cfg, W, row[:-1], torch.float32)[69:].argmax(-1).tolist()
    _status_clean()
