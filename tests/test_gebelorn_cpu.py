"""The Gebelorn design on the CPU path in fp32: configuration, weights, cache, scheduler, portions and decoding against
the plain statement in ``gebelorn_oracle``."""
import io
import json
import math

import pytest
import torch

import gebelorn_cases as cases
import gebelorn_oracle as oracle
from pisceslx_b200 import YvConfig
from pisceslx_b200.models.cache import RELEASED, YvCacheConfig, YvPagedLayeredCache
from pisceslx_b200.models.latent_attention import rotary_for
from pisceslx_b200.ops import latent as L

TOL = 2e-5


@pytest.fixture(scope="module")
def mixed():
    cfg = cases.mixed()
    W = cases.weights(cfg)
    toks = cases.tokens(cfg, 210)
    return cfg, W, cases.build(cfg, W), toks, cases.expected(cfg, W, toks)


@pytest.mark.parametrize("name", sorted(cases.CUTS))
def test_any_cut_of_a_sequence_gives_the_plain_logits(mixed, name):
    cfg, W, m, toks, want = mixed
    got = cases.run_cut(cases.engine(m), 0, toks, cases.CUTS[name])
    assert cases.error(got, want).max() < TOL


def test_sizes_no_vector_divides():
    cfg = cases.odd()
    W = cases.weights(cfg, 3)
    m, toks = cases.build(cfg, W), cases.tokens(cfg, 90)
    want = cases.expected(cfg, W, toks)
    for cuts in ([1000], [1], [7, 1, 2]):
        assert cases.error(cases.run_cut(cases.engine(m), 0, toks, cuts), want).max() < TOL


def test_stream_after_every_layer(mixed):
    cfg, W, m, toks, _ = mixed
    ref = []
    cases.expected(cfg, W, toks[:40], layers_out=ref)
    seen = []
    m.model.layer_tap = lambda i, x: seen.append((i, x.clone()))
    try:
        m(input_ids=torch.tensor([toks[:40]]))
    finally:
        m.model.layer_tap = None
    assert [i for i, _ in seen] == [0, 1, 2]
    for (_, x), r in zip(seen, ref):
        assert (x - r.float()).abs().max() < 1e-4 * r.abs().max()


def test_without_token_side_and_window():
    cfg = cases.mixed()
    del cfg["token_side"]
    del cfg["layers"][1]["mixer"]["mask"]
    W = cases.weights(cfg, 5)
    m, toks = cases.build(cfg, W), cases.tokens(cfg, 90)
    eng = cases.engine(m)
    assert eng.cache.reach is None                   # one layer reads everything: no page may go
    assert cases.error(cases.run_cut(eng, 0, toks, [30, 1]), cases.expected(cfg, W, toks)).max() < TOL


@pytest.mark.parametrize("scaling", [None, cases.YARN, {"factor": 8.0, "original": 1000, "fast": 32.0, "slow": 1.0},
                                     {"factor": 0.5, "original": 30, "fast": 9.0, "slow": 0.01}])
@pytest.mark.parametrize("dims", [2, 10, 32])
def test_rotation_tables(scaling, dims):
    rot = {"dims": dims, "base": 5000.0}
    spec = dict(rot)
    if scaling:
        rot["scaling"] = scaling
        spec["yarn"] = scaling
    cos, sin = rotary_for(spec).tables(3000, torch.device("cpu"))
    x = torch.randn(dims, dtype=torch.float64, generator=torch.Generator().manual_seed(dims))
    from pisceslx_b200.ops import reference as ref
    for pos in (0, 1, 17, 2999):
        got = ref.apply_rope(x.view(1, 1, -1).float(), cos, sin, torch.tensor([pos]), dims).view(-1)
        assert torch.allclose(got, oracle.rotate(x, pos, rot).float(), atol=3e-6)
    if scaling:                                      # the end of the ramp may lie past the last pair
        freq, mag = oracle.rotary_frequencies(rot)
        assert math.isclose(mag, 0.1 * math.log(scaling["factor"]) + 1.0) and len(freq) == dims // 2


def _edge_case(window, T, far, d=8, r=4, vd=8):
    """Keys that do not matter, except that position ``far`` would take all the weight of every query that sees it."""
    g = torch.Generator().manual_seed(T + far)
    q = torch.zeros(T, d + r)
    q[:, 0] = 1.0
    k = 0.01 * torch.randn(T, d, generator=g)
    k[far, 0] = 60.0
    return q, k, torch.randn(T, vd, generator=g), 0.01 * torch.randn(T, r, generator=g)


@pytest.mark.parametrize("window", [1, 2, 64, 65])
def test_window_edge_is_exact(window):
    T, far = 150, 20
    q, k, v, kr = _edge_case(window, T, far)
    cu = torch.tensor([0, T], dtype=torch.int32)
    got = L.latent_attention(q, k, v, kr, None, cu, cu, T, 1, window, 1.0)
    for t in range(T):
        inside = far <= t < far + window
        assert torch.allclose(got[t], v[far], atol=1e-3) == inside, (t, inside)


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [(1, 4, 2, 3, 9, None), (3, 8, 4, 5, 12, 6), (2, 5, 6, 4, 7, 1)])
def test_decode_in_the_latent_space_equals_attention_over_keys_and_values(heads, dim, rot, vdim, rank, window):
    g = torch.Generator().manual_seed(11)
    B, bs, lens = 3, 4, [1, 9, 14]
    rnd = lambda *s: torch.randn(*s, generator=g)
    w_uk, w_uv, cache, q = rnd(heads, dim, rank), rnd(heads, vdim, rank), rnd(16, bs, rank + rot), rnd(B, heads * (dim + rot))
    gate = rnd(B, heads)
    table = torch.randperm(16, generator=g)[:12].view(3, 4).int()
    pos = torch.tensor([n - 1 for n in lens], dtype=torch.int32)
    rotspec = {"dims": rot, "base": 50.0}
    cos, sin = rotary_for(rotspec).tables(64, torch.device("cpu"))
    q_lat = L.latent_query_absorbed(q, w_uk.transpose(1, 2).contiguous(), rot, cos, sin, pos)
    o_lat = L.latent_decode(q_lat, cache, rank, table, torch.tensor(lens, dtype=torch.int32), window, 0.7)
    got = L.latent_values(o_lat, w_uv, gate, B).view(B, heads, vdim)
    for b, n in enumerate(lens):
        js = oracle.visible(n - 1, n, window)
        rows = torch.stack([cache[table[b, j // bs], j % bs] for j in js])
        qb = q[b].view(heads, dim + rot)
        kn = torch.einsum("hdr,jr->jhd", w_uk, rows[:, :rank])
        v = torch.einsum("hdr,jr->jhd", w_uv, rows[:, :rank])
        want = oracle.attend(qb[:, :dim], oracle.rotate(qb[:, dim:], n - 1, rotspec), kn, rows[:, rank:], v, 0.7)
        assert torch.allclose(got[b], want * torch.sigmoid(gate[b])[:, None], atol=1e-4)


def test_norm_activation_and_token_gate():
    g = torch.Generator().manual_seed(2)
    x, y, w, w2 = (torch.randn(*s, generator=g) for s in ((5, 12), (5, 12), (12,), (12,)))
    stream = x.clone()
    h = L.stream_norm(stream, y, w, w2, 1e-3, torch.float32)
    want = x + oracle.rms(y, w, 1e-3)
    assert torch.allclose(stream, want, atol=1e-6) and torch.allclose(h, oracle.rms(want, w2, 1e-3), atol=1e-5)
    z = torch.linspace(-6, 6, 101)
    assert torch.allclose(L.gelu(z), oracle.gelu_erf(z), atol=1e-6)
    table, ids = torch.randn(9, 30, generator=g), torch.tensor([0, 8, 3, 3, 1])
    a = torch.randn(5, 7, generator=g)
    assert torch.allclose(L.token_gate(a, table, 14, ids), oracle.gelu_tanh(a) * table[ids][:, 14:21], atol=1e-6)


def test_pages_behind_every_window_are_given_back_and_used_again(mixed):
    cfg, W, m, toks, want = mixed
    eng = cases.engine(m, blocks=10, block_size=16)
    free0 = eng.cache.alloc.available()
    eng.cache.add_sequence(7)
    got = []
    for at in range(0, 210, 3):
        got.append(eng.run_tokens(7, toks[at:at + 3], [0, 1, 2]))
        held = [b for b in eng.cache.tables[7] if b != RELEASED]
        # widest window 70: at most 69 tokens before the portion, the portion, one page of slack and two partial pages
        assert len(held) <= (69 + 3) // 16 + 3
    assert len(set(eng.cache.tables[7])) > 1 and eng.cache.tables[7][0] == RELEASED
    assert cases.error(torch.cat(got), want).max() < TOL     # 210 tokens went through 10 pages of 16
    eng.cache.free_sequence(7)
    assert eng.cache.alloc.available() == free0
    # the same pages serve another sequence at once
    other = cases.tokens(cfg, 60, seed=9)
    assert cases.error(cases.run_cut(eng, 8, other, [13, 1]), cases.expected(cfg, W, other)).max() < TOL


def test_cache_rows_state_round_trip_and_fork():
    c = YvPagedLayeredCache([{"row": 6}, {"row": 10}], YvCacheConfig(block_size=4, num_blocks=8, dtype=torch.float32), torch.device("cpu"), reach=5)
    c.add_sequence(1)
    slots = c.append_slots(1, 12)
    assert list(c.slots(1, 0, 12)) == slots
    c.rows(1).view(-1, 10)[slots[9]] = 3.0
    c.append_slots(1, 8)
    assert c.tables[1][0] == RELEASED and c.alloc.available() == 8 - 4
    with pytest.raises(IndexError):
        c.slots(1, 0, 4)
    c.fork(1, 2)
    c.free_sequence(1)
    assert c.alloc.available() == 8 - 4
    st = c.state()
    d = YvPagedLayeredCache([{"row": 6}, {"row": 10}], c.cfg, c.device, reach=5)
    d.load_state(st)
    assert d.tables == c.tables and d.alloc.available() == 4 and d.rows(1).view(-1, 10)[slots[9], 0] == 3.0
    d.free_sequence(2)
    assert d.alloc.available() == 8


def test_batches_of_unequal_requests_and_greedy_generation_through_the_scheduler(mixed):
    cfg, W, m, _, _ = mixed
    prompts = [cases.tokens(cfg, n, seed=20 + n) for n in (1, 5, 64, 97, 33)]
    new = [9, 30, 4, 12, 21]

    def plain(prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(cases.expected(cfg, W, seq)[-1].argmax()))
        return seq[len(prompt):]

    want = [plain(p, n) for p, n in zip(prompts, new)]
    for kw in ({}, {"prefill_portion": 13}, {"max_num_seqs": 2}):
        eng = cases.engine(m, blocks=30, block_size=16, **kw)
        reqs = [eng.add_request(p, max_new_tokens=n) for p, n in zip(prompts, new)]
        eng.run_until_done()
        assert [r.output_ids for r in reqs] == want, kw
        assert eng.cache.alloc.available() == 30


def test_generate_entry_point_batches_equal_prompts(mixed):
    cfg, W, m, toks, _ = mixed
    ids = torch.tensor([toks[:20], toks[40:60]])
    out, stats = m.generate(ids, max_new_tokens=6)
    assert stats["generated_tokens"] == 6
    for row, start in zip(out.tolist(), (toks[:20], toks[40:60])):
        for i in range(20, 26):
            assert row[i] == int(cases.expected(cfg, W, row[:i])[-1].argmax())


def _write_folder(path, cfg, W, dtype_name="BF16"):
    (path / "config.json").write_text(json.dumps(cfg))
    header, blob = {"__metadata__": {"made": "by a test"}}, b""
    for k, v in W.items():
        raw = v.contiguous().view(torch.uint8).numpy().tobytes()
        header[k] = {"dtype": dtype_name, "shape": list(v.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    hd = json.dumps(header).encode()
    (path / "model.safetensors").write_bytes(len(hd).to_bytes(8, "little") + hd + blob)


def test_checkpoint_folder_decides_class_sizes_and_weights(tmp_path, mixed):
    from pisceslx_b200.engine.loader import load_model_for_inference, save_pretrained
    from pisceslx_b200.models.layered import YvLayeredForCausalLM
    cfg, W, m, toks, want = mixed
    _write_folder(tmp_path, cfg, W)
    m2 = load_model_for_inference(ckpt=str(tmp_path), device="cpu", dtype=torch.float32)
    assert isinstance(m2, YvLayeredForCausalLM) and m2.cfg.vocab_size == cfg["vocab"] and m2.cfg.n_layer == 3
    assert cases.error(cases.run_cut(cases.engine(m2), 0, toks[:50], [50]), want[:50]).max() < TOL
    # the framework's own save format and the configuration's round trip
    save_pretrained(m2, str(tmp_path / "saved"))
    m3 = load_model_for_inference(ckpt=str(tmp_path / "saved"), device="cpu", dtype=torch.float32)
    for (k, a), b in zip(sorted(m2.checkpoint_slices().items()), (v for _, v in sorted(m3.checkpoint_slices().items()))):
        assert torch.equal(a, b), k
    assert YvConfig.from_dict(m2.cfg.to_dict()).to_dict() == m2.cfg.to_dict()
    n = sum(v.numel() for v in W.values())
    assert m2.cfg.count_parameters()["total"] == n


def test_bad_checkpoints_are_refused(tmp_path):
    cfg = cases.odd()
    W = cases.weights(cfg)
    m = cases.build(cfg, W)
    with pytest.raises(KeyError):
        m.load_reference_state_dict({k: v for k, v in W.items() if k != "l1.mix.uk"})
    with pytest.raises(ValueError):
        m.load_reference_state_dict({**W, "head": W["head"][:-1]})
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError):
        YvConfig.from_dict(bad)
    with pytest.raises(ValueError):
        YvConfig.from_dict({"architecture": "NoSuchDesign"})
    from pisceslx_b200.engine.weights import read_safetensors
    _write_folder(tmp_path, cfg, W)
    raw = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "model.safetensors").write_bytes(raw[:-7])
    with pytest.raises(ValueError):
        read_safetensors(tmp_path / "model.safetensors")


def test_trace_replay_steps_ends_and_order(mixed, tmp_path):
    import numpy as np
    from pisceslx_b200.serve.trace import YvTraceReplayer
    cfg, W, m, toks, want = mixed
    eng = cases.engine(m, blocks=12)
    free0 = eng.cache.alloc.available()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:9], "want": [8, 0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[9:80], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[80:81], "want": [0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "a", "tokens": toks[:2], "want": [1]}], "end": ["a"]}]
    out = io.StringIO()
    YvTraceReplayer(eng, str(tmp_path)).run(io.StringIO("\n".join(map(json.dumps, steps)) + "\n"), out)
    assert out.getvalue().splitlines() == ["done 0", "done 1", "done 2", "done 5"]
    assert eng.cache.alloc.available() == free0 and not (tmp_path / "1.f32").exists()
    for n, pos in ((0, [8, 0, 8]), (2, [80]), (5, [1])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(len(pos), cfg["vocab"]).copy())
        assert cases.error(got, want[pos]).max() < TOL


def test_command_line_generates_from_a_checkpoint_folder(tmp_path, capsys):
    import manage
    cfg = cases.odd()
    cfg["vocab"] = 300
    _write_folder(tmp_path, cfg, cases.weights(cfg))
    assert manage.main(["infer", "--model_path", str(tmp_path), "--device", "cpu", "--dtype", "fp32", "--prompt", "abc",
                        "--max_new_tokens", "4"]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["stats"]["generated_tokens"] == 4


def test_a_planted_mistake_shows():
    """The comparison is sharp enough: an oracle with one wrong constant is told apart at once."""
    cfg = cases.mixed()
    W = cases.weights(cfg)
    toks = cases.tokens(cfg, 110)
    good = cases.expected(cfg, W, toks)
    for change in (lambda m: m["mask"].__setitem__("size", m["mask"]["size"] + 1),
                   lambda m: m["mask"].__setitem__("size", m["mask"]["size"] - 1),
                   lambda m: m.__setitem__("scale", m["scale"] * 1.01),
                   lambda m: m["rot"].__setitem__("base", m["rot"]["base"] * 1.1)):
        bad = json.loads(json.dumps(cfg))
        change(bad["layers"][1]["mixer"])
        assert cases.error(cases.expected(bad, W, toks), good).max() > 20 * TOL
