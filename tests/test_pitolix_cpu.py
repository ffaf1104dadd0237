"""The Pitolix design on the CPU path in fp32: configuration, weights, layer loop, cache, scheduler, portions and decoding
against the plain statement in ``pitolix_oracle``."""
import io
import json

import pytest
import torch

import pitolix_cases as cases
import pitolix_oracle as oracle
from pisceslx_b200 import YvConfig
from pisceslx_b200.models.cache import YvCacheConfig, YvPagedLayeredCache
from pisceslx_b200.models.latent_attention import rotary_for
from pisceslx_b200.models.registry import cache_layout, kernel_families
from pisceslx_b200.ops import grouped as G
from pisceslx_b200.ops import latent as L

TOL = 2e-5


@pytest.fixture(scope="module")
def mixed():
    cfg = cases.mixed()
    W = cases.weights(cfg)
    toks = cases.tokens(cfg, 210)
    return cfg, W, cases.build(cfg, W), toks, cases.expected(cfg, W, toks)


# ---- the model -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(cases.CUTS))
def test_any_cut_of_a_sequence_gives_the_plain_logits(mixed, name):
    cfg, W, m, toks, want = mixed
    got = cases.run_cut(cases.engine(m), 0, toks, cases.CUTS[name])
    assert cases.error(got, want).max() < TOL


@pytest.mark.parametrize("make", [cases.odd, cases.wide, cases.plain])
def test_other_sizes(make):
    cfg = make()
    W = cases.weights(cfg, 3)
    m, toks = cases.build(cfg, W), cases.tokens(cfg, 90)
    want = cases.expected(cfg, W, toks)
    for cuts in ([1000], [1], [7, 1, 2]):
        assert cases.error(cases.run_cut(cases.engine(m), 0, toks, cuts), want).max() < TOL


def test_stream_after_every_run_of_a_layer(mixed):
    cfg, W, m, toks, _ = mixed
    ref, seen = [], []
    cases.expected(cfg, W, toks[:40], layers_out=ref)
    m.model.layer_tap = lambda i, x: seen.append((i, x.clone()))
    try:
        m(input_ids=torch.tensor([toks[:40]]))                       # without a cache: keys and values in packed rows
    finally:
        m.model.layer_tap = None
    assert [i for i, _ in seen] == list(range(1 + 3 * 2 + 1))
    for (_, x), r in zip(seen, ref):
        assert (x - r.float()).abs().max() < 1e-4 * r.abs().max()


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (0, 4, 2), (0, 1, 3), (3, 4, 2), (1, 4, 2)])
def test_loops_anywhere(loop):
    """Order of the runs, their caches, and what is added in front of each pass, also at the first and the last layer."""
    cfg = cases.mixed()
    cfg.pop("loop")
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    c = YvConfig.from_dict(cfg)
    assert c.layer_runs() == oracle.order(cfg)
    assert len(cache_layout(c)[0]) == len(oracle.order(cfg)) and cache_layout(c)[1] is None
    W = cases.weights(cfg, 5)
    m, toks = cases.build(cfg, W), cases.tokens(cfg, 40)
    assert cases.error(cases.run_cut(cases.engine(m), 0, toks, [9, 1, 4, 2]), cases.expected(cfg, W, toks)).max() < TOL


def test_every_pass_has_its_own_cache(mixed):
    cfg, _, m, toks, _ = mixed
    eng = cases.engine(m)
    eng.cache.add_sequence(0)
    eng.run_tokens(0, toks[:20], [0])
    k = [eng.cache.layer(r)[0] for r in (1, 3, 5)]                    # layer 1 in its three passes
    assert k[0].shape == k[1].shape and not torch.allclose(k[0], k[1]) and not torch.allclose(k[1], k[2])


# ---- mechanisms, each alone ------------------------------------------------------------------------------------------
def _run_mixer(kind, mx, T=40, width=48, seed=1, change=None):
    g = torch.Generator().manual_seed(seed)
    cfg = cases.config([{"type": kind, "mixer": mx, "mlp": None}], vocab=8, width=width, eps=1e-3)
    W = cases.weights(cfg, seed)
    if change:
        change(W)
    m = cases.build(cfg, W)
    h = torch.randn(T, width, generator=g)
    ctx = m.model.build_context(1, T, torch.device("cpu"))
    blk = m.model.layers[0]
    z = torch.empty(T, blk.mixer.out_width)
    blk.mixer.attend(h, ctx, 0, z)
    got = z @ blk.out_proj[:, :blk.mixer.out_width].T
    want = oracle.mixer(kind, h.double(), {k: v.double() for k, v in W.items()}, "l0.mix.", mx, 1e-3)
    return got, want


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,temp", [(6, 2, 16, 8, (0.5, 7)), (4, 4, 9, 13, (0.3, 1)), (5, 1, 8, 24, None)])
def test_normed_attention_alone(heads, kv_heads, dim, vdim, temp):
    got, want = _run_mixer("attention", cases.normed(heads, kv_heads, dim, vdim, None, 1.7, temp)["mixer"])
    assert torch.allclose(got.double(), want, atol=1e-5)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims", [(6, 2, 16, 8, 16), (4, 4, 10, 13, 4), (3, 1, 24, 8, 2)])
def test_rotated_attention_alone(heads, kv_heads, dim, vdim, dims):
    got, want = _run_mixer("attention_2", cases.rotated(heads, kv_heads, dim, vdim, None, 0.4, dims)["mixer"])
    assert torch.allclose(got.double(), want, atol=1e-5)


def test_a_sink_takes_the_weight_it_stands_for():
    """A sink far above the scores leaves nothing, one far below changes nothing."""
    mx = cases.normed(2, 1, 8, 8, None, 1.0)["mixer"]
    big, _ = _run_mixer("attention", mx, change=lambda W: W["l0.mix.sink"].fill_(60.0))
    none, want = _run_mixer("attention", mx, change=lambda W: W["l0.mix.sink"].fill_(-60.0))
    assert big.abs().max() < 1e-12 and none.abs().max() > 0.1 and torch.allclose(none.double(), want, atol=1e-5)


@pytest.mark.parametrize("every", [1, 2, 16, 64])
def test_temperature_steps_at_the_right_positions(every):
    """Constant before the step's first position, one step higher from there on."""
    T, temp = 70, {"coef": 0.9, "every": every}
    q = torch.ones(T, 4)
    pages = torch.zeros(T, 1, 1, 4)
    G.grouped_prep(q, torch.ones(T, 4), torch.ones(T, 4), None, [0, 0, 0], 1, 1, pages, pages.clone(), None,
                   torch.arange(T, dtype=torch.int32), None, None, 0, False, temp, 1e-6)
    for t in range(T):
        assert abs(q[t, 0].item() - oracle.temperature(t, temp)) < 1e-6
    assert (q[every - 1, 0] > 1.0) and (every == 1 or q[every - 2, 0] == 1.0)


@pytest.mark.parametrize("dims,dim", [(2, 2), (6, 9), (32, 32)])
def test_partial_rotation(dims, dim):
    rot = {"dims": dims, "base": 5000.0}
    cos, sin = rotary_for(rot).tables(3000, torch.device("cpu"))
    g = torch.Generator().manual_seed(dims)
    pos = torch.tensor([0, 1, 17, 2999], dtype=torch.int32)
    q, k, v = torch.randn(4, 2 * dim, generator=g), torch.randn(4, dim, generator=g), torch.randn(4, 3, generator=g)
    kp, vp, q0 = torch.zeros(4, 1, 1, dim), torch.zeros(4, 1, 1, 3), q.clone()
    G.grouped_prep(q, k, v, None, [0, 0, 0], 2, 1, kp, vp, None, pos, cos, sin, dims, False, None, 1e-6)
    for t, p in enumerate(pos.tolist()):
        assert torch.allclose(q[t].view(2, dim), oracle.rotate(q0[t].view(2, dim).double(), p, rot).float(), atol=3e-6)
        assert torch.allclose(kp[t, 0], oracle.rotate(k[t].view(1, dim).double(), p, rot).float(), atol=3e-6)
    assert torch.equal(vp.view(4, 3), v)


def test_joins_norms_and_activation():
    g = torch.Generator().manual_seed(2)
    T, C = 5, 12
    x, w, w2, vec = (torch.randn(*s, generator=g) for s in ((T, C), (C,), (C,), (C,)))
    parts, table, ids = torch.randn(3, T + 2, C, generator=g), torch.randn(9, C, generator=g), torch.tensor([0, 8, 3, 3, 1])
    s = x.clone()
    h1, h2 = L.stream_add(s, parts, (w, w2), 1.0, 1e-3, torch.float32, table=table, rows=ids, table_scale=2.5, vec=vec)
    want = x + parts[:, :T].sum(0) + 2.5 * table[ids] + vec
    assert torch.allclose(s, want, atol=1e-5)
    assert torch.allclose(h1, oracle.norm(want, w, 1e-3), atol=1e-5) and torch.allclose(h2, oracle.norm(want, w2, 1e-3), atol=1e-5)
    assert L.stream_add(s, None, (), 1.0, 1e-3, torch.float32, table=table, rows=ids, start=True) == ()
    assert torch.allclose(s, table[ids])
    W = {"m.gate": torch.randn(7, C, generator=g), "m.up": torch.randn(7, C, generator=g), "m.down": torch.eye(7)}
    out = torch.empty(T, 9)
    L.swiglu(torch.cat([x @ W["m.gate"].T, x @ W["m.up"].T], 1), out[:, 1:8])
    assert torch.allclose(out[:, 1:8], oracle.feed_forward(x, W, "m."), atol=1e-5)


@pytest.mark.parametrize("far", [0, 1, 63, 64, 127])
def test_a_standing_out_key_is_seen_from_its_own_position_on(far):
    """Causal to the position: one key takes all the weight of every query that sees it, through pages out of order."""
    T, d, bs = 150, 8, 16
    g = torch.Generator().manual_seed(far)
    q, k, v = torch.zeros(T, 2 * d), 0.01 * torch.randn(T, d, generator=g), torch.randn(T, d, generator=g)
    q[:, 0] = q[:, d] = 1.0
    k[far, 0] = 60.0
    table = torch.randperm(12, generator=g)[:-(-T // bs)].int().view(1, -1)
    kp, vp = torch.full((12, bs, 1, d), 9.0), torch.full((12, bs, 1, d), 9.0)
    slots = torch.tensor([int(table[0, t // bs]) * bs + t % bs for t in range(T)])
    kp.view(-1, d)[slots], vp.view(-1, d)[slots] = k, v
    for n in (2, 50, T):                                              # the last n positions as a portion
        out = torch.empty(n, 2 * d)
        G.grouped_attention(q[T - n:], kp, vp, table, torch.tensor([T]), torch.tensor([0, n]), n, 2, 1.0, None, None, out)
        for i in range(n):
            assert torch.allclose(out[i, :d], v[far], atol=1e-3) == (far <= T - n + i), (n, i)


# ---- cache and scheduler ---------------------------------------------------------------------------------------------
def test_pages_are_used_again_by_another_sequence(mixed):
    cfg, W, m, toks, want = mixed
    eng = cases.engine(m, blocks=14, block_size=16)
    free0 = eng.cache.alloc.available()
    assert cases.error(cases.run_cut(eng, 7, toks, [50, 1, 3, 1]), want).max() < TOL
    assert eng.cache.alloc.available() == free0
    for t in eng.cache.k + eng.cache.v:
        t.mul_(100.0)                                                 # whatever the pages still hold must not matter
    other = cases.tokens(cfg, 60, seed=9)
    assert cases.error(cases.run_cut(eng, 8, other, [13, 1]), cases.expected(cfg, W, other)).max() < TOL


def test_interleaved_sequences_keep_apart(mixed):
    cfg, W, m, toks, want = mixed
    other = cases.tokens(cfg, 90, seed=4)
    eng = cases.engine(m, blocks=24, block_size=16)
    got = {0: [], 1: []}
    for s in (0, 1):
        eng.cache.add_sequence(s)
    for at in range(0, 90, 5):
        for s, seq in ((0, toks), (1, other)):
            got[s].append(eng.run_tokens(s, seq[at:at + 5], [0, 1, 2, 3, 4]))
    assert cases.error(torch.cat(got[0]), want[:90]).max() < TOL
    assert cases.error(torch.cat(got[1]), cases.expected(cfg, W, other)).max() < TOL


def test_cache_layouts_state_round_trip_and_fork():
    layouts = [{"row": 6}, {"heads": 2, "dim": 3, "vdim": 5}]
    c = YvPagedLayeredCache(layouts, YvCacheConfig(block_size=4, num_blocks=8, dtype=torch.float32), torch.device("cpu"))
    assert c.rows(0).shape == (8, 4, 6) and c.layer(1)[0].shape == (8, 4, 2, 3) and c.layer(1)[1].shape == (8, 4, 2, 5)
    with pytest.raises(TypeError):
        c.rows(1)
    with pytest.raises(TypeError):
        c.layer(0)
    assert c.bytes() == 32 * (6 + 6 + 10) * 4
    c.add_sequence(1)
    slots = c.append_slots(1, 9)
    c.layer(1)[1].view(-1, 10)[slots[8]] = 3.0
    c.fork(1, 2)
    c.free_sequence(1)
    d = YvPagedLayeredCache(layouts, c.cfg, c.device)
    d.load_state(c.state())
    assert d.tables == c.tables and d.layer(1)[1].view(-1, 10)[slots[8], 0] == 3.0
    d.free_sequence(2)
    assert d.alloc.available() == 8


def test_batches_of_unequal_requests_and_greedy_generation_through_the_scheduler(mixed):
    cfg, W, m, _, _ = mixed
    prompts = [cases.tokens(cfg, n, seed=20 + n) for n in (1, 5, 64, 97, 33)]
    new = [9, 20, 4, 8, 15]

    def plain(prompt, n):
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(cases.expected(cfg, W, seq, torch.float32)[-1].argmax()))
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
    for row in out.tolist():
        want = cases.expected(cfg, W, row[:-1])[19:].argmax(-1).tolist()
        assert row[20:] == want


# ---- configuration, weights, command line ----------------------------------------------------------------------------
def _write_folder(path, cfg, W):
    (path / "config.json").write_text(json.dumps(cfg))
    header, blob = {}, b""
    for k, v in W.items():
        raw = v.contiguous().view(torch.uint8).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    hd = json.dumps(header).encode()
    (path / "model.safetensors").write_bytes(len(hd).to_bytes(8, "little") + hd + blob)


def test_checkpoint_folder_decides_class_sizes_and_weights(tmp_path, mixed):
    from pisceslx_b200.engine.loader import load_model_for_inference, save_pretrained
    from pisceslx_b200.models.layered import YvLayeredForCausalLM
    cfg, W, m, toks, want = mixed
    _write_folder(tmp_path, cfg, W)
    m2 = load_model_for_inference(ckpt=str(tmp_path), device="cpu", dtype=torch.float32)
    assert isinstance(m2, YvLayeredForCausalLM) and m2.cfg.vocab_size == cfg["vocab"] and m2.cfg.n_layer == 4
    assert cases.error(cases.run_cut(cases.engine(m2), 0, toks[:50], [50]), want[:50]).max() < TOL
    save_pretrained(m2, str(tmp_path / "saved"))
    m3 = load_model_for_inference(ckpt=str(tmp_path / "saved"), device="cpu", dtype=torch.float32)
    for (k, a), b in zip(sorted(m2.checkpoint_slices().items()), (v for _, v in sorted(m3.checkpoint_slices().items()))):
        assert torch.equal(a, b), k
    assert YvConfig.from_dict(m2.cfg.to_dict()).to_dict() == m2.cfg.to_dict()
    assert m2.cfg.count_parameters()["total"] == sum(v.numel() for v in W.values())
    assert kernel_families(m2.cfg) == ("grouped_attention",)


@pytest.mark.parametrize("make", [cases.odd, cases.plain])
def test_parameter_count(make):
    cfg = make()
    assert YvConfig.from_dict(cfg).count_parameters()["total"] == sum(v.numel() for v in cases.weights(cfg).values())


def test_bad_checkpoints_and_configurations_are_refused():
    cfg = cases.odd()
    W = cases.weights(cfg)
    m = cases.build(cfg, W)
    with pytest.raises(KeyError):
        m.load_reference_state_dict({k: v for k, v in W.items() if k != "l1.mix.k.b"})
    with pytest.raises(ValueError):
        m.load_reference_state_dict({**W, "l0.mix.sink": W["l0.mix.sink"][:-1]})
    for change in (lambda c: c["layers"][0].__setitem__("type", "something_else"),
                   lambda c: c["layers"][0]["mlp"].__setitem__("kind", "sparse"),
                   lambda c: c.__setitem__("loop", {"start": 1, "stop": 4, "times": 2}),
                   lambda c: c.__setitem__("loop", {"start": 1, "stop": 1, "times": 2})):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            YvConfig.from_dict(bad)


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
    """The comparison is sharp enough: an oracle with one wrong constant or weight is told apart at once."""
    cfg = cases.mixed()
    W = cases.weights(cfg)
    toks = cases.tokens(cfg, 60)
    good = cases.expected(cfg, W, toks)
    mixers = [e["mixer"] for e in cfg["layers"]]
    for where, key, value in ((mixers[1]["q_temp"], "every", 17), (mixers[1]["q_temp"], "coef", 0.41),
                              (mixers[0], "scale", 0.303), (mixers[2]["rot"], "base", 220.0), (mixers[2]["rot"], "dims", 14),
                              (cfg["embedding"], "scale", 2.51), (cfg["loop"], "times", 2), (cfg["norm"], "eps", 3e-2)):
        old, where[key] = where[key], value
        assert cases.error(cases.expected(cfg, W, toks), good).max() > 20 * TOL, key
        where[key] = old
    for name in ("l1.mix.sink", "l0.mix.q.b", "l2.mix.v.b", "loop.step", "l3.mix.g"):
        bad = dict(W)
        bad[name] = torch.zeros_like(W[name])
        assert cases.error(cases.expected(cfg, bad, toks), good).max() > 20 * TOL, name
