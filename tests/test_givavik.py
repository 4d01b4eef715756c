"""Givavik through the framework's own step function, cache manager, scheduler and kernels, against the plain model of
``plain_givavik.py``.  Model-level cases run twice: on the host with plain Python standing in for the kernels (what is
under test there is the plan, the parts' wiring, the shared latents, the states of blocks and embedding, the cache
manager and the packer), and on a GPU with the kernels themselves.  Kernel-level cases compare each new kernel with its
restatement in ``plain_ops.py`` at sizes of their own, or with a value that is known by construction."""
import math

import numpy as np
import pytest
import torch

import givavik_util as gu
import plain_givavik as plain
import plain_ops
import vukavik_util as vu           # the schedule runner and the error measures are not tied to a model


@pytest.fixture()
def kernels(monkeypatch):
    """On the host the plain restatements stand in for the kernels; on a GPU nothing is replaced."""
    def use(device):
        if device == "cpu":
            from vapi_b200 import ops
            for name in plain_ops.ALL:
                monkeypatch.setattr(ops, name, getattr(plain_ops, name))
    return use


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg, seed in [("mixed", gu.MIXED, 1), ("tiny", gu.TINY, 2), ("plain", gu.PLAIN, 3), ("serving_heads", gu.SERVING_HEADS, 4)] + \
            [(k, v, 10 + i) for i, (k, v) in enumerate(gu.ONE.items())]:
        out[name] = gu.write_model(str(tmp_path_factory.mktemp(name)), cfg, seed)
        out[name + "/bf16"] = gu.write_model(str(tmp_path_factory.mktemp(name + "bf16")), cfg, seed, torch.bfloat16)
    return out


_oracles = {}


def _oracle(folder):
    return _oracles.setdefault(folder, gu.Oracle(folder))


def _check(runner, oracle, requests, schedule, dtype):
    got = vu.run_schedule(runner, requests, schedule)
    for rid, toks in requests.items():
        want = oracle.logits(toks)
        e = np.abs(got[rid] - want.numpy()).max(-1) / float(want.max() - want.min())
        gu.within(e, oracle.rounding(toks, dtype), dtype, f"request {rid}", vu.limit(dtype))


def _close(a, b, tol):
    a, b = a.float().cpu(), b.float().cpu()
    assert torch.isfinite(a).all()
    assert float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), f"{float((a - b).abs().max()):.3e}"


# ---- configuration, registry and what a request keeps ---------------------------------------------------------
def test_the_architecture_is_found_by_its_name_and_every_size_comes_from_the_configuration():
    from vapi_b200.config.model import ConfigError, resolve_architecture
    from vapi_b200.parts import LatentAttention, ParallelMixer
    arch = resolve_architecture(gu.MIXED)
    assert arch.name == "Givavik"
    plan = arch.plan(arch.parse(gu.MIXED))
    shapes = {s.name: tuple(s.shape) for s in plan.tensor_specs()}
    assert shapes["embed"] == (200, 64) and shapes["bigram"] == (38, 64) and shapes["head"] == (200, 64) and shapes["final.norm"] == (64,)
    assert shapes["l0.mix.left.q"] == (64, 64) and shapes["l0.mix.left.k"] == (32, 64) and shapes["l0.mix.left.v"] == (48, 64)
    assert shapes["l0.mix.left.q.b"] == (64,) and shapes["l0.mix.left.o"] == (64, 96) and shapes["l0.mix.left.o.b"] == (64,)
    assert shapes["l0.mix.left.pb"] == (4,) and shapes["l0.shift"] == (64,) and shapes["l0.ls2"] == (64,)
    assert shapes["l0.mix.right.in"] == (2 * 60 + 2 * 3 * 20 + 6, 64) and shapes["l0.mix.right.conv"] == (60 + 120, 3)
    assert shapes["l0.mix.right.o"] == (64, 60) and shapes["l0.mlp.up"] == (72, 64) and shapes["l0.mlp.act"] == (2,)
    assert shapes["l1.mix.q"] == (3 * 20, 64) and shapes["l1.mix.dkv"] == (32, 64) and shapes["l1.mix.dkv.norm"] == (24,)
    assert shapes["l1.mix.uk"] == (36, 24) and shapes["l1.mix.uv"] == (60, 24) and shapes["l1.mix.sink"] == (3,) and shapes["l1.mix.o"] == (64, 60)
    assert shapes["l2.mix.q"] == (2 * 28, 64) and shapes["l2.mix.uk"] == (40, 24) and "l2.mix.dkv" not in shapes and "l2.mix.dkv.norm" not in shapes
    assert "l2.ls2" not in shapes and not any(k.startswith("l2.mlp") for k in shapes), "a layer without a feed-forward"
    assert "l0.mix.left.q_norm" not in shapes and not any("layernorm" in k for k in shapes), "q and k are normed without a weight"
    assert [c.cache_of for c in plan.order] == [None, None, 1, None, None, 1]
    # every layer keeps its last normed row, also one that reads another's latents; the embedding keeps a token
    sites = dict(plan.cache_sites())
    assert {k for k in sites if isinstance(k, tuple) and k[0] == "block"} == {("block", i) for i in range(6)}
    assert sites["embedding"].dtype == torch.int32 and all(sites[("block", i)].shape == (64,) for i in range(6))
    assert set(sites) == {"embedding", 1, 4, (0, 0), (0, 1), (3, 0), (3, 1)} | {("block", i) for i in range(6)}
    assert [type(b.mixer) for b in plan.layers] == [ParallelMixer, LatentAttention, LatentAttention, ParallelMixer, LatentAttention, LatentAttention]
    le, ri = plan.layers[3].mixer.branches
    assert (le.nh, le.nkv, le.d, le.dv, le.scale, le.softcap, le.rot_dim, le.weights, le.qk_norm_eps) == (3, 3, 24, 16, 0.2, 0.9, 24, "sigmoid", 1e-5)
    assert (ri.nh, ri.p, ri.N, ri.G, ri.L, ri.norm_groups) == (2, 40, 12, 1, 5, 4) and plan.layers[3].mixer.factors == [1.3, 0.6]
    assert len(plan.position_encodings) == 4, "rotary tables are shared only by layers that agree on them"
    assert plan.embedding.scale == 1.7 and plan.embedding.bigram == ("bigram", 37, 91, 13)
    free = arch.plan(arch.parse(gu.PLAIN))
    assert free.embedding.bigram is None and "embedding" not in dict(free.cache_sites()) and free.layers[0].mixer.branches[0].softcap == 0.0
    lat = gu.layer(gu.latent())
    for bad in ([{"type": "attention", "mixer": {}, "mlp": None}],
                [gu.layer(gu.parallel(gu.left(heads=3, kv_heads=2)))],
                [gu.layer(gu.parallel(gu.left(dims=18)))],
                [gu.layer(gu.parallel(gu.left(softcap=-1.0)))],
                [gu.layer(gu.parallel(None, gu.right(heads=5, groups=2)))],
                [gu.layer(gu.parallel(None, gu.right(norm_groups=7)))],
                [gu.layer(gu.latent(kv_from=0))],                                               # itself
                [lat, gu.layer(gu.latent(kv_from=0)), gu.layer(gu.latent(kv_from=1))],          # a layer without a latent of its own
                [lat, gu.layer(gu.latent(kv_from=0, kv_rank=28))], [lat, gu.layer(gu.latent(kv_from=0, base=7.0))],
                [gu.layer(gu.parallel()), gu.layer(gu.latent(kv_from=0))],
                [{**lat, "mlp": {"kind": "moe", "ff": 8}}]):
        with pytest.raises(ConfigError):
            arch.parse({**gu.MIXED, "layers": bad})


def test_states_of_unlike_types_share_a_slot(folders, kernels):
    kernels("cpu")
    r = vu.make_runner(folders["tiny"], "float32", "cpu", num_pages=4)
    kinds = {g.spec.kind: g.tensor.dtype for g in r.cache.state}
    assert kinds == {"previous_token": torch.int32, "token_shift": torch.float32, "mamba2": torch.float32}
    assert [v.block.tensor.shape for v in r.views(type("C", (), {"groups": [None] * 4})())] == [(5, 32)] * 3
    r = vu.make_runner(folders["tiny"], "bfloat16", "cpu", num_pages=4)
    assert {g.spec.kind: g.tensor.dtype for g in r.cache.state} == kinds, "what the recurrences carry is 32-bit whatever the dtype"


# ---- the plain model itself, by hand ---------------------------------------------------------------------------
def test_the_plain_mechanisms_by_hand():
    f64 = lambda *v: torch.tensor(v, dtype=torch.float64)
    # the second table: the row of a pair of tokens, and the last row for a first token
    assert plain.bigram_row(3, 5, {"mul_prev": 7, "mul_cur": 2, "buckets": 10}) == (21 + 10) % 10
    cfg = {"embedding": {"scale": 2.0, "bigram": {"mul_prev": 7, "mul_cur": 2, "buckets": 10}}}
    w = {"embed": torch.eye(6, dtype=torch.float64), "bigram": torch.arange(11, dtype=torch.float64)[:, None] * torch.ones((1, 6), dtype=torch.float64)}
    x = plain.embedding(cfg, w, [3, 5])
    assert float(x[0, 3]) == 12.0 and float(x[0, 0]) == 10.0 and float(x[1, 5]) == 3.0 and float(x[1, 0]) == 1.0
    # the shift: nothing before the first token, a part of the token before afterwards, element by element
    h = torch.tensor([[2.0, 4.0], [6.0, 8.0]], dtype=torch.float64)
    assert torch.equal(plain.token_shift(h, f64(0.25, 1.0)), torch.tensor([[1.5, 0.0], [5.0, 4.0]], dtype=torch.float64))
    # a norm weight of zero changes nothing
    assert torch.allclose(plain.zero_centred_norm(f64(3.0, 4.0), f64(0.0, 1.0), 0.0), f64(3.0, 8.0) / math.sqrt(12.5))
    # interleaved pairs
    r = plain.rotate_pairs(f64(1, 2, 3, 4, 5), 3, 4, 10.0)
    a1 = 3.0 * 10.0 ** -0.5
    assert float(r[0]) == pytest.approx(math.cos(3) - 2 * math.sin(3)) and float(r[1]) == pytest.approx(2 * math.cos(3) + math.sin(3))
    assert float(r[2]) == pytest.approx(3 * math.cos(a1) - 4 * math.sin(a1)) and float(r[4]) == 5.0
    # xIELU on both sides of zero, and continuous there
    act = f64(0.3, -0.4)
    sp = lambda v: math.log1p(math.exp(v))
    y = plain.xielu(f64(2.0, -1.5, 0.0), act)
    assert float(y[0]) == pytest.approx(sp(0.3) * 4 + 1.0) and float(y[2]) == 0.0
    assert float(y[1]) == pytest.approx((0.5 + sp(-0.4)) * (math.exp(-1.5) - 1 + 1.5) - 0.75)
    # sigmoid attention: one key of capped score s has the weight sigmoid(s + b), and two equal keys count twice
    eye, z2 = torch.eye(2, dtype=torch.float64), torch.zeros(2, dtype=torch.float64)
    wa = {"q": eye, "k": eye, "v": eye, "o": eye, "q.b": z2, "k.b": z2, "v.b": z2, "o.b": f64(0.5, 0.0), "pb": f64(-0.7)}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 3.0, "softcap": 2.0}
    s = torch.tensor([[1.0, 2.0], [1.0, 2.0]], dtype=torch.float64)
    out = plain.sigmoid_attention(wa, "", m, s, 0.0)
    sc = 2.0 * math.tanh(3.0 * 2.0 / 2.0)                            # q and k are unit in the mean square, so q.k = 2
    wgt = 1 / (1 + math.exp(-(sc - 0.7)))
    assert torch.allclose(out, torch.stack([wgt * s[0], 2 * wgt * s[0]]) + f64(0.5, 0.0))
    # a sink takes its share of one key's weight: exp(s) / (exp(s) + exp(sink))
    wl = {"q": torch.ones((1, 1), dtype=torch.float64), "uk": torch.ones((1, 1), dtype=torch.float64),
          "uv": torch.ones((1, 1), dtype=torch.float64), "o": torch.ones((1, 1), dtype=torch.float64), "sink": f64(0.4)}
    ml = {"heads": 1, "dim": 1, "rot_dim": 0, "vdim": 1, "kv_rank": 1, "scale": 1.0, "rot": {"base": 1.0, "dims": 0}}
    out = plain.latent_attention(wl, "", ml, torch.tensor([[1.5]], dtype=torch.float64), torch.ones((1, 1), dtype=torch.float64),
                                 torch.zeros((1, 0), dtype=torch.float64))
    assert float(out) == pytest.approx(math.exp(1.5) / (math.exp(1.5) + math.exp(0.4)))
    # Mamba-2 from zero: the first token's state is its own write, the second decays it
    wm = {"in": torch.tensor([[0.0], [1.0], [1.0], [1.0], [0.0]], dtype=torch.float64), "conv": torch.tensor([[0.0, 1.0]] * 3, dtype=torch.float64),
          "conv.b": torch.zeros(3, dtype=torch.float64), "dt_bias": f64(0.0), "A_log": f64(0.0), "D": f64(0.0), "norm": f64(1.0), "o": torch.eye(1, dtype=torch.float64)}
    mm = {"heads": 1, "vdim": 1, "state": 1, "groups": 1, "conv": 2, "norm_groups": 1}
    assert torch.equal(plain.mamba2(wm, "", mm, torch.tensor([[1.0], [1.0]], dtype=torch.float64), 1.0), torch.zeros((2, 1), dtype=torch.float64)), "silu(0) shuts the gate"


# ---- the model against the plain one: whole prompts, decoding, portions -----------------------------------------
WHOLE = [pytest.param("cpu", "tiny", [19], id="host"),
         pytest.param("cuda", "mixed", [150, 1, 37], marks=pytest.mark.gpu, id="gpu-mixed"),
         pytest.param("cuda", "plain", [70, 2], marks=pytest.mark.gpu, id="gpu-plain"),
         pytest.param("cuda", "serving_heads", [100], marks=pytest.mark.gpu, id="gpu-serving-heads"),
         pytest.param("cuda", "latent", [40], marks=pytest.mark.gpu, id="gpu-latent-alone"),
         pytest.param("cuda", "parallel", [40], marks=pytest.mark.gpu, id="gpu-parallel-alone"),
         pytest.param("cuda", "shared", [40], marks=pytest.mark.gpu, id="gpu-shared-latents")]


@pytest.mark.parametrize("device,name,lens", WHOLE)
def test_whole_prompt_token_by_token_and_portions_agree_with_the_plain_model(device, name, lens, folders, kernels):
    """Each request alone: its whole prompt in one step; a prompt and then single tokens; portions of changing size
    down to two tokens, cut inside pages and where a shift, a bigram and a convolution reach over the cut."""
    kernels(device)
    oracle = _oracle(folders[name])
    runner = vu.make_runner(folders[name], "float32", device, num_pages=12)
    for i, n in enumerate(lens):
        toks = gu.prompt(oracle.cfg, n, 20 + i)
        _check(runner, oracle, {"a": toks}, [[("a", n)]], "float32")
        head = max(1, n - 12) if device == "cuda" else max(1, n - 4)
        _check(runner, oracle, {"b": toks}, [[("b", head)]] + [[("b", 1)]] * (n - head), "float32")
        if n > 2:
            _check(runner, oracle, {"c": toks}, [[("c", q)] for q in vu.cuts(n, [2, 3, 17, 5, 64, 2, 16, 1])], "float32")
            _check(runner, oracle, {"d": toks}, [[("d", q)] for q in vu.cuts(n, [16, 15, 2, 31])], "float32")


@pytest.mark.gpu
def test_long_decoding_one_token_at_a_time(folders):
    """Every token alone from the first: 170 steps through the caches and every state."""
    oracle = _oracle(folders["mixed"])
    runner = vu.make_runner(folders["mixed"], "float32", "cuda", num_pages=12)
    toks = gu.prompt(oracle.cfg, 170, 5)
    _check(runner, oracle, {"a": toks}, [[("a", 1)]] * 170, "float32")


BATCH = [pytest.param("cpu", "tiny", "float32", [7, 1, 12, 3, 9], 16, id="host"),
         pytest.param("cuda", "mixed", "float32", [70, 1, 33, 150, 2, 64, 17], 16, marks=pytest.mark.gpu, id="gpu-f32"),
         pytest.param("cuda", "mixed/bf16", "bfloat16", [70, 1, 33, 150, 2, 64, 17], 16, marks=pytest.mark.gpu, id="gpu-bf16"),
         pytest.param("cuda", "serving_heads/bf16", "bfloat16", [150, 40, 3, 86, 70], 64, marks=pytest.mark.gpu, id="gpu-bf16-tensor-cores"),
         pytest.param("cuda", "plain/bf16", "bfloat16", [60, 5, 31], 16, marks=pytest.mark.gpu, id="gpu-bf16-plain")]


@pytest.mark.parametrize("device,name,dtype,lens,page", BATCH)
def test_unequal_requests_in_one_batch_match_each_alone(device, name, dtype, lens, page, folders, kernels):
    """More requests than state slots and a pool smaller than their sum: portions of some beside single tokens of
    others, requests that pause, pages and slots that pass from finished requests to new ones; then the same
    schedule once more on the same runner, over whatever the first pass left in pages and slots."""
    kernels(device)
    oracle = _oracle(folders[name])
    need = sorted((-(-n // page) for n in lens), reverse=True)
    runner = vu.make_runner(folders[name], dtype, device, num_pages=sum(need[:4]) + 1, page_size=page, max_requests=4, max_tokens=512)
    reqs = {f"r{i}": gu.prompt(oracle.cfg, n, 40 + i) for i, n in enumerate(lens)}
    g = torch.Generator().manual_seed(3)
    left = {k: len(v) for k, v in reqs.items()}
    waiting, live, schedule = list(reqs), [], []
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for rid in list(live):
            if len(live) > 1 and float(torch.rand(1, generator=g)) < 0.2:
                continue                                        # left out of this step, goes on later
            q = min(left[rid], int(torch.tensor([1, 1, 2, 3, 16, 29, 70])[torch.randint(0, 7, (1,), generator=g)]))
            step.append((rid, q))
            left[rid] -= q
            if left[rid] == 0:
                live.remove(rid)
        if step:
            schedule.append(step)
    for _ in range(2):
        _check(runner, oracle, reqs, schedule, dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "serving_heads"])
def test_how_a_prompt_is_cut_and_what_else_runs_changes_rounding_only(name, folders):
    """bfloat16: the same request whole, in portions, and in a batch with others, against itself."""
    cfg = gu.MIXED if name == "mixed" else gu.SERVING_HEADS
    page = 64
    runner = vu.make_runner(folders[name + "/bf16"], "bfloat16", "cuda", num_pages=12, page_size=page, max_tokens=512)
    toks, other = gu.prompt(cfg, 140, 1), gu.prompt(cfg, 120, 2)
    a = vu.run_schedule(runner, {"a": toks}, [[("a", 140)]])["a"]
    span = float(a.max() - a.min())
    for schedule in ([[("a", q)] for q in vu.cuts(140, [2, 63, 65, 7])], [[("b", 50), ("a", 100)]] + [[("a", 1), ("b", 1)]] * 40 + [[("b", 30)]]):
        reqs = {"a": toks, "b": other} if any(r == "b" for st in schedule for r, _ in st) else {"a": toks}
        b = vu.run_schedule(runner, reqs, schedule)["a"]
        d = np.abs(a - b).max(-1) / span
        assert d.max() < 0.04 and d.mean() < 0.008, f"{d.max():.3e} {d.mean():.3e}"


# ---- the new kernels against their restatements -------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [64, 99, 324, 2048, 4096, 4100])
def test_the_shift_rides_on_the_norm(hidden, dtype):
    """Pending outputs, norm and token shift in one kernel: first tokens of fresh requests (whatever their slots hold),
    first tokens of a portion, single tokens and long portions; the new stream in memory of its own; every last row
    left in its slot and the other slots alone.  700 tokens: a block takes several rows one after another."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(hidden)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    sa, sb, w, sh = (torch.randn(hidden, generator=g) for _ in range(4))
    c = lambda t: None if t is None else t.cuda()
    for lens, starts in (([1], [0]), ([1], [7]), ([3, 1, 2, 9, 1], [0, 0, 5, 64, 3]), ([400, 1, 4, 295, 3], [0, 9, 2, 100, 0])):
        n = sum(lens)
        cu, seq, pos, slots = gu.step_index(lens, starts, [6, 0, 3, 4, 1][:len(lens)])
        x = torch.randn((n, hidden), generator=g) * 3.0
        ya, yb = (torch.randn((n, hidden), generator=g).to(dtype) for _ in range(2))
        state = torch.randn((8, 2, hidden), generator=g)
        for a, s1, b, s2, both in ((ya, sa, yb, sb, True), (ya, sa, None, None, True), (ya, None, yb, sb, False), (None, None, None, None, True)):
            want_state, got_state = state.clone(), state.clone().cuda()
            want = plain_ops.shift_add_rmsnorm(x, a, s1, b, s2, w, 1e-6, sh, want_state[:, 1], slots, seq, cu, pos, dtype, plain=both)
            xd = x.cuda()
            got = ops.shift_add_rmsnorm(xd, c(a), c(s1), c(b), c(s2), w.cuda(), 1e-6, sh.cuda(), got_state[:, 1], slots.cuda(), seq.cuda(),
                                        cu.cuda(), pos.cuda(), dtype, plain=both)
            assert torch.equal(xd.cpu(), x), "the stream that was handed in is not written"
            for gt, wt, tl in zip(got, want, (1e-6, tol, tol)):
                assert (gt is None) == (wt is None)
                if wt is not None:
                    _close(gt, wt, tl)
            _close(got_state, want_state, 2e-5)
            others = [i for i in range(8) if i not in slots.tolist()]
            assert torch.equal(got_state.cpu()[others], state[others]) and torch.equal(got_state.cpu()[:, 0], state[:, 0])


@pytest.mark.gpu
def test_cutting_a_sequence_changes_no_bit_of_its_shift():
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(1)
    n, H = 65, 256
    x, y = torch.randn((n, H), generator=g).cuda(), torch.randn((n, H), generator=g).cuda()
    w, sh = torch.randn(H, generator=g).cuda(), torch.rand(H, generator=g).cuda()

    def run(cuts):
        state, outs, at = torch.full((2, H), 9.0).cuda(), [], 0
        for q in cuts:
            cu, seq, pos, slots = (t.cuda() for t in gu.step_index([q], [at], [1]))
            outs.append(ops.shift_add_rmsnorm(x[at:at + q].contiguous(), y[at:at + q].contiguous(), None, None, None, w, 1e-5, sh, state, slots,
                                              seq, cu, pos, torch.float32)[2])
            at += q
        return torch.cat(outs), state[1].clone()
    whole = run([n])
    for cuts in ([1] * n, [2, 2, 31, 30], [64, 1], [1, 64]):
        got = run(cuts)
        assert torch.equal(got[0], whole[0]) and torch.equal(got[1], whole[1])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_bigram_rows_and_the_token_they_carry(dtype):
    """Fresh requests (the last row), portions that go on (the token before comes from the slot), products beyond 32
    bits, a single bucket; the slots move on and nobody else's is touched."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(3)
    for V, H, buckets, mp, mc in ((50, 40, 17, 5, 3), (70000, 132, 1009, 99991, 31337), (9, 64, 1, 4, 7), (300, 1024, 4096, 1, 0)):
        table, big = torch.randn((V, H), generator=g).to(dtype), torch.randn((buckets + 1, H), generator=g).to(dtype)
        lens, starts = [5, 1, 1, 300, 2], [0, 0, 9, 64, 3]
        cu, seq, pos, slots = gu.step_index(lens, starts, [2, 6, 0, 5, 3])
        toks = torch.randint(0, V, (sum(lens),), generator=g, dtype=torch.int32)
        state = torch.randint(0, V, (8, 1), generator=g, dtype=torch.int32)
        want_state, got_state = state.clone(), state.clone().cuda()
        want = plain_ops.embed_bigram(table, big, toks, pos, seq, cu, want_state, slots, mp, mc, 0.37)
        got = ops.embed_bigram(table.cuda(), big.cuda(), toks.cuda(), pos.cuda(), seq.cuda(), cu.cuda(), got_state, slots.cuda(), mp, mc, 0.37)
        _close(got, want, 1e-6)
        assert torch.equal(got_state.cpu(), want_state)
        first = table[int(toks[0])].float() * 0.37 + big[buckets].float()
        assert torch.allclose(got[0].cpu(), first, atol=1e-5)
    with pytest.raises(ops.KernelError):
        ops.embed_bigram(table.cuda(), big.cuda()[:, :8].contiguous(), toks.cuda(), pos.cuda(), seq.cuda(), cu.cuda(), got_state, slots.cuda(), 1, 1)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_xielu_alone_and_behind_a_product(dtype):
    """Elementwise at sizes that are no multiple of four, values from far below zero to far above, both sides of zero;
    then as the epilogue of every product that takes it (1 to 16, 17 to 32 and prompt-sized steps) and behind the library's."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(7)
    consts = torch.tensor([0.83, 1.21])
    z = torch.cat([torch.linspace(-30, 30, 2001), torch.tensor([0.0, -1e-4, 1e-4, -1e-2, 1e-2])])[:, None].to(dtype)
    _close(ops.xielu(z.cuda(), consts.cuda()), plain_ops.xielu(z.float(), consts).to(dtype), 1e-6 if dtype == torch.float32 else 8e-3)
    near = z[-5:].float()
    got = ops.xielu(near.cuda(), consts.cuda()).cpu()
    assert torch.allclose(got, plain_ops.xielu(near.double(), consts.double()).float(), rtol=1e-4, atol=1e-9), "digits are kept next to zero"
    for n, K, N in ((1, 64, 40), (7, 96, 136), (16, 320, 72), (20, 64, 200), (32, 192, 136), (100, 64, 96), (256, 128, 200), (300, 72, 264), (1030, 64, 72)):
        x, w = (torch.randn((n, K), generator=g)).to(dtype), (torch.randn((N, K), generator=g) * 0.2).to(dtype)
        want = plain_ops.xielu(x.float() @ w.float().t(), consts)
        got = ops.linear_xielu(x.cuda(), w.cuda(), consts.cuda())
        assert got.dtype == dtype and got.shape == (n, N)
        _close(got, want, 2e-5 if dtype == torch.float32 else 2e-2)
        if dtype == torch.bfloat16 and n > 32:
            _close(ops.prompt_linear(w.cuda(), act=x.cuda(), epilogue="bf16", xielu=consts.cuda()), want, 2e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_interleaved_latent_rows_with_the_queries_riding_along(dtype):
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(11)
    for n, R, r, rot, H, d, page in ((9, 24, 8, 8, 3, 12, 4), (70, 200, 64, 32, 5, 40, 16), (1, 4, 4, 4, 1, 4, 8), (33, 512, 64, 64, 2, 128, 64)):
        down = torch.randn((n, R + r), generator=g) * 2.0
        wc = torch.randn(R, generator=g)
        pos = torch.randint(0, 5000, (n,), generator=g)
        freq = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
        cos, sin = torch.cos(pos[:, None].float() * freq), torch.sin(pos[:, None].float() * freq)
        pages = -(-n // page) + 2
        slots = torch.randperm(pages * page, generator=g)[:n].to(torch.int32)
        cache = torch.randn((pages, page * (R + r)), generator=g).to(dtype)
        q = torch.randn((n, H * (d + r)), generator=g).to(dtype)
        full = torch.full((n, H, R + r), 5.0).to(dtype)
        want_c, want_f, got_c, got_f = cache.clone(), full.clone(), cache.cuda(), full.cuda()
        kw = dict(interleaved=True, heads=H, dim=d)
        assert plain_ops.latent_prepare(down, 0, R, r, None, wc, 1e-5, cos, sin, rot, want_c, page, slots, dtype, q=q, qfull=want_f, **kw) is None
        assert ops.latent_prepare(down.cuda(), 0, R, r, None, wc.cuda(), 1e-5, cos.cuda(), sin.cuda(), rot, got_c, page, slots.cuda(), dtype,
                                  q=q.cuda(), qfull=got_f, **kw) is None
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        _close(got_c, want_c, tol)
        _close(got_f, want_f, tol)
        assert bool((got_f[:, :, :R] == 5.0).all()), "the unrotated part is the batched product's"
        alone = full.cuda()
        ops.latent_rotate_q(q.cuda(), alone, H, d, r, R, cos.cuda(), sin.cuda(), rot, interleaved=True)
        assert torch.equal(alone, got_f)
        # by hand: the pair (2i, 2i + 1) of the shared key part
        t, i = n - 1, rot // 2 - 1
        u, v = float(down[t, R + 2 * i]), float(down[t, R + 2 * i + 1])
        row = got_c.cpu().view(pages * page, R + r)[int(slots[t])].float()
        assert float(row[R + 2 * i]) == pytest.approx(u * float(cos[t, i]) - v * float(sin[t, i]), abs=0.05 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_sink_in_the_shared_cache(dtype):
    """One cached row of score s: a head returns exp(s) / (exp(s) + exp(sink)) of it, on both kernels (widths of 16n take
    the tensor cores in bfloat16) and counted once however the keys are split; then a mixed batch against the restatement."""
    from vapi_b200 import ops
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for R, r in ((24, 8), (32, 16), (128, 32)):
        H, page = 3, 16
        sinks = torch.tensor([-3.0, 0.5, 40.0])
        for s in (-2.0, 3.0):
            cache = torch.zeros((2, page * (R + r)))
            cache[1, :R] = 1.0
            cache[1, R:R + r] = 1.0
            q = torch.zeros((1, H, R + r))
            q[:, :, R] = s
            idx = [t.cuda() for t in (torch.tensor([[1]], dtype=torch.int32), torch.tensor([0, 1], dtype=torch.int32), torch.tensor([1], dtype=torch.int32))]
            for splits in (1, 4):
                out = ops.latent_attention(q.view(1, -1).to(dtype).cuda(), cache.to(dtype).cuda(), page, *idx, 1, 1, 1, 1, H, R, r, 1.0,
                                           splits=splits, sinks=sinks.cuda()).float().cpu().view(H, R)
                for h in range(H):
                    assert torch.allclose(out[h], torch.full((R,), 1.0 / (1.0 + math.exp(float(sinks[h]) - s))), atol=1e-2 if dtype == torch.bfloat16 else 1e-6)
    g = torch.Generator().manual_seed(2)
    for H, R, r, page in ((5, 36, 4, 8), (3, 64, 16, 16), (4, 96, 16, 64), (2, 256, 32, 8), (2, 512, 64, 16)):
        lens, klens = [1, 9, 30, 2], [150, 9, 41, 33]
        cache, table, cu, sk = gu.batch(lens, klens, page, R + r, H * R, dtype)
        n = sum(lens)
        q = (torch.randn((n, H * (R + r)), generator=g) * 0.3).to(dtype)
        sinks = torch.randn(H, generator=g) * 2.0
        args = (n, 4, max(lens), max(klens), H, R, r, 0.2)
        want = plain_ops.latent_attention(q, cache, page, table, cu, sk, *args, sinks=sinks)
        for splits in (1, 3):
            got = ops.latent_attention(q.cuda(), cache.cuda(), page, table.cuda(), cu.cuda(), sk.cuda(), *args, splits=splits, sinks=sinks.cuda())
            _close(got, want, tol)


# keys and values of one width of 64 or 128 on pages of 64: the tensor cores for bfloat16 (portions of 64 tokens and more
# at width 64 on the tcgen05 kernel); everything else on the general kernel
HEADS = [(20, 12, 8), (64, 64, 64), (128, 128, 64), (64, 64, 16), (256, 96, 16)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dk,dv,page", HEADS)
def test_sigmoid_weights_on_every_attention_kernel(dtype, dk, dv, page):
    """A mixed batch against the restatement: no cap, a cap far above the scores (where tanh is a polynomial on the
    tensor cores), a cap that flattens them; a score bias per head; a factor on the output; into rows of their own and
    into columns of a wider buffer; keys split and not."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(dk + dv)
    nh, nkv = 6, 2
    tol = 3e-5 if dtype == torch.float32 else 1.5e-2
    for lens, klens in (([1, 9, 2, 1], [150, 9, 66, 64]), ([70, 1, 33], [70, 130, 65]), ([129], [150])):
        n, S = sum(lens), len(lens)
        cache, table, cu, sk = gu.batch(lens, klens, page, nkv * (dk + dv), dk, dtype, spread=1.0)
        q = torch.randn((n, nh * dk + 8), generator=g).to(dtype)
        bias = torch.randn(nh, generator=g) * 2.0 - 1.0
        for scale, cap, b, f in ((0.3, 0.0, bias, 1.0), (0.5 / dk ** 0.5, 30.0, bias, 0.7), (2.0, 3.0, None, 1.3)):
            args = (n, S, max(lens), max(klens), nh, nkv, dk, dv, scale)
            kw = dict(weights="sigmoid", softcap=cap, out_scale=f)
            want = plain_ops.masked_attention(q, nh * dk + 8, cache, page, table, cu, sk, *args, score_bias=b, **kw)
            dev = (q.cuda(), nh * dk + 8, cache.cuda(), page, table.cuda(), cu.cuda(), sk.cuda()) + args
            db = None if b is None else b.cuda()
            _close(ops.masked_attention(*dev, score_bias=db, splits=1, **kw), want, tol)
            if max(lens) < 64:
                _close(ops.masked_attention(*dev, score_bias=db, splits=3, **kw), want, tol)
            for wide, at in ((nh * dv + 24, 0), (nh * dv + 10, 4)):
                buf = torch.full((n, wide), 9.0, dtype=dtype).cuda()
                ops.masked_attention(*dev, score_bias=db, out=buf[:, at:at + nh * dv], **kw)
                _close(buf[:, at:at + nh * dv], want, tol)
                assert bool((buf[:, :at] == 9.0).all()) and bool((buf[:, at + nh * dv:] == 9.0).all()), "the rest of the buffer is someone else's"
    with pytest.raises(ops.KernelError):
        ops.masked_attention(*dev, weights="sigmoid", sinks=torch.zeros(nh).cuda())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dk,dv,page", HEADS)
def test_a_far_key_is_found_by_its_sigmoid(dtype, dk, dv, page):
    """One key among hundreds whose weight is near one where all the others' are near nothing: far back, at page borders,
    the newest key, the first, just behind the query; for single tokens, with split keys, and in portions of every size
    that picks another kernel."""
    from vapi_b200 import ops
    nh, nkv = 4, 2
    for klen, j_star, qlen, splits in ((900, 3, 1, 1), (900, 3, 1, 4), (900, 63, 1, 2), (900, 64, 7, 3), (641, 640, 1, 2), (640, 639, 1, 1),
                                       (333, 0, 40, 1), (130, 63, 99, 1), (130, 64, 99, 1), (97, 96, 33, 2), (200, 127, 128, 1),
                                       (200, 128, 128, 1), (2, 0, 2, 1), (1, 0, 1, 1), (64, 63, 64, 1)):
        cache, table, cu, sk = gu.batch([qlen], [klen], page, nkv * (dk + dv), klen + j_star, torch.float32, spread=0.01)
        pg, off = int(table[0, j_star // page]), j_star % page
        for h in range(nkv):
            cache[pg, (h * page + off) * dk] = 10.0
            v0 = nkv * page * dk + (h * page + off) * dv
            cache[pg, v0:v0 + dv] = 1.0
        q = torch.zeros((qlen, nh * dk))
        q[:, ::dk] = 2.0                                         # score 20 for the planted key, near zero for the others
        out = ops.masked_attention(q.to(dtype).cuda(), nh * dk, cache.to(dtype).cuda(), page, table.cuda(), cu.cuda(), sk.cuda(), qlen, 1, qlen,
                                   klen, nh, nkv, dk, dv, 1.0, weights="sigmoid", softcap=40.0,
                                   score_bias=torch.full((nh,), -10.0).cuda(), splits=splits).float().cpu()
        want = 1.0 / (1.0 + math.exp(-(40.0 * math.tanh(0.5) - 10.0)))
        for j in range(qlen):
            seen = j_star <= klen - qlen + j
            assert bool(((out[j] - (want if seen else 0.0)).abs() < 0.05).all()), f"keys {klen}, planted {j_star}, query at {klen - qlen + j}, splits {splits}"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_cap_and_a_bias_before_a_softmax(dtype):
    """The same options with the softmax (the general kernel), split and not, with a sink."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(6)
    nh, nkv = 4, 2
    for dk, dv, page in ((20, 12, 8), (64, 64, 64)):
        lens, klens = [1, 9, 70], [90, 9, 75]
        n = sum(lens)
        cache, table, cu, sk = gu.batch(lens, klens, page, nkv * (dk + dv), dk, dtype, spread=1.0)
        q = torch.randn((n, nh * dk), generator=g).to(dtype)
        kw = dict(softcap=2.5, score_bias=torch.randn(nh, generator=g), sinks=torch.randn(nh, generator=g), out_scale=1.5)
        args = (n, 3, max(lens), max(klens), nh, nkv, dk, dv, 0.4)
        want = plain_ops.masked_attention(q, nh * dk, cache, page, table, cu, sk, *args, **kw)
        dkw = {k: v.cuda() if torch.is_tensor(v) else v for k, v in kw.items()}
        for splits in (1, 3):
            got = ops.masked_attention(q.cuda(), nh * dk, cache.cuda(), page, table.cuda(), cu.cuda(), sk.cuda(), *args, splits=splits, **dkw)
            _close(got, want, 3e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_gated_norm_writes_into_a_wider_buffer(dtype):
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(8)
    for n, width, groups in ((5, 96, 3), (40, 1536, 2)):
        y, z, w = torch.randn((n, width), generator=g), torch.randn((n, width + 8), generator=g).to(dtype), torch.randn(width, generator=g)
        want = plain_ops.gated_group_rmsnorm(y, z[:, 4:4 + width], w, 1e-5, width // groups, True, dtype)
        buf = torch.full((n, width + 40), 7.0, dtype=dtype).cuda()
        ops.gated_group_rmsnorm(y.cuda(), z.cuda()[:, 4:4 + width], w.cuda(), 1e-5, width // groups, True, dtype, out=buf[:, 32:32 + width])
        _close(buf[:, 32:32 + width], want, 2e-5 if dtype == torch.float32 else 2e-2)
        assert bool((buf[:, :32] == 7.0).all()) and bool((buf[:, 32 + width:] == 7.0).all())


@pytest.mark.parametrize("device,dtype", [pytest.param("cpu", torch.float32, id="host"), pytest.param("cuda", torch.float32, marks=pytest.mark.gpu, id="gpu")])
def test_joined_projections_are_the_branches_with_their_factors(device, dtype, folders, kernels):
    """The two mixers of a layer through their joint products against each alone through its own, factors applied by hand."""
    kernels(device)
    from vapi_b200.engine.step import StepEntry
    name = "tiny" if device == "cpu" else "mixed"
    layer_at = 1 if device == "cpu" else 0
    r = vu.make_runner(folders[name], "float32", device, num_pages=8)
    rc = r.cache.open("a")
    n = 11
    assert r.cache.reserve(rc, n)
    ctx = r.packer.pack([StepEntry(rc, gu.prompt({"vocab": r.vocab_size}, n, 3), [])], dtype, status=r.status)
    for pe in r.plan.position_encodings:
        ctx.pos[pe.name] = pe.prepare(ctx)
    view = r.views(ctx)[layer_at]
    mixer = r.plan.layers[layer_at].mixer
    a = torch.randn((n, r.plan.hidden_size), generator=torch.Generator().manual_seed(1)).to(device)
    joint = mixer.forward(a, ctx, view)
    assert mixer.branches[0].w_qkv is None and mixer.branches[1].w_o is None, "nobody keeps the projections twice"
    from vapi_b200.config.model import load_config_json, resolve_architecture
    from vapi_b200.weights.loader import load_tensors
    cfg = load_config_json(folders[name])
    arch = resolve_architecture(cfg)
    again = arch.plan(arch.parse(cfg))
    tensors = load_tensors(folders[name], again.tensor_specs(), dtype, device)
    alone = torch.zeros_like(a)
    for sub, m, f, v in zip(("left.", "right."), again.layers[layer_at].mixer.branches, mixer.factors, view.parts):
        m.bind(tensors, f"l{layer_at}.mix." + sub, dtype)
        alone += f * m.forward(a, ctx, v)
    _close(joint, alone, 1e-5)
    from vapi_b200.parts import GQAttention, ParallelMixer, ShortConv
    with pytest.raises(ValueError):
        ParallelMixer(8, [("a.", ShortConv(8, 3))], factors=(1.0, 2.0))
    assert GQAttention(64, 4, 2, 16).pieces() is None, "the plain form of attention keeps its specialised kernels"


# ---- the engine: scheduler, batching, sampling, entry point -----------------------------------------------------
@pytest.mark.parametrize("device,name,lens,new", [pytest.param("cpu", "tiny", [1, 9, 20], 5, id="host"),
                                                  pytest.param("cuda", "mixed", [1, 33, 80, 7, 64, 40], 10, marks=pytest.mark.gpu, id="gpu")])
def test_greedy_generation_through_the_entry_point(device, name, lens, new, folders, kernels):
    """More requests than slots, prompts cut into portions of 16 beside other requests' decoding; on a GPU pure
    decode steps run as captured graphs, one step ahead of the host (the token before is then known to the device
    alone).  Slots and pages pass from finished requests to waiting ones."""
    kernels(device)
    from vapi_b200 import LLM, SamplingParams
    oracle = _oracle(folders[name])
    llm = LLM(folders[name], dtype="f32", device=device, num_blocks=40, page_size=16, max_concurrent_seqs=4,
              max_batched_tokens=64, prefill_chunk_tokens=16, max_context=256, cuda_graphs=device == "cuda")
    prompts = [gu.prompt(oracle.cfg, n, 50 + i) for i, n in enumerate(lens)]
    out = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True))
    for p, c in zip(prompts, out):
        want = oracle.greedy(p, new)
        if c.tokens != want:                 # only a near-tie of the plain model's own logits may part them
            i = next(k for k in range(new) if c.tokens[k] != want[k])
            top = torch.topk(oracle.logits(list(p) + want[:i])[-1], 2).values
            assert float(top[0] - top[1]) < 1e-3, f"prompt of {len(p)}: token {i} differs without a tie"
    llm.runner.cache.check_invariants()


@pytest.mark.gpu
def test_preempted_requests_start_over(folders):
    """A pool too small for the requests that were admitted: some are put back and computed again from position 0, in
    slots that hold what others left."""
    from vapi_b200 import LLM, SamplingParams
    oracle = _oracle(folders["mixed"])
    prompts = [gu.prompt(oracle.cfg, n, 80 + i) for i, n in enumerate([28, 30, 25, 31])]
    llm = LLM(folders["mixed"], dtype="f32", device="cuda", num_blocks=11, page_size=16, max_concurrent_seqs=4, max_batched_tokens=64,
              max_context=128, cuda_graphs=False)
    out = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, c in zip(prompts, out):
        logits = oracle.logits(list(p) + c.tokens[:-1])
        for i, t in enumerate(c.tokens):
            row = logits[len(p) - 1 + i]
            assert float(row.max() - row[t]) < 1e-3, f"prompt of {len(p)}: token {i} is not the plain model's choice"


# ---- trace replay: the program a user replays a trace with ----------------------------------------------------------
def _trace(cfg):
    import replay_util as rp
    reqs = {f"r{i}": gu.prompt(cfg, n, 70 + i) for i, n in enumerate([1, 70, 40, 90, 66])}
    tr = rp.Trace()
    rp.whole(tr, "w", reqs["r1"])
    rp.tail_decode(tr, "t", reqs["r2"], tail=5)
    rp.portions(tr, "p", reqs["r3"], sizes=[2, 3, 61, 2, 1])
    mix = {f"m{k}": v for k, v in reqs.items()}
    rp.mixed(tr, mix, seed=5, decode_tail=3)
    return tr, {"w": reqs["r1"], "t": reqs["r2"], "p": reqs["r3"], **mix}


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_as_a_user_runs_it(dtype, folders, tmp_path):
    """The replay program as a child process: four state slots and a pool for the live requests only."""
    import replay_util as rp
    name = "mixed" if dtype == "float32" else "mixed/bf16"
    oracle = _oracle(folders[name])
    tr, tokens = _trace(oracle.cfg)
    got = rp.run_trace(folders[name], dtype, tr, str(tmp_path / "out"))
    ref = {k: oracle.logits(v).float() for k, v in tokens.items()}
    span = max(float(r.max() - r.min()) for r in ref.values())
    where = [(step, i, rid, pos) for step, rows in tr.rows.items() for i, (rid, pos) in enumerate(rows)]
    e = [np.abs(got[step][i] - ref[rid][pos].numpy()).max() / span for step, i, rid, pos in where]
    slack = [oracle.rounding(tokens[rid], dtype)[pos] for _, _, rid, pos in where]
    gu.within(e, slack, dtype, "replay", vu.limit(dtype))
