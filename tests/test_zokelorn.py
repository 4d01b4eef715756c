"""Zokelorn through the framework's own step function, cache manager, scheduler and kernels, against the plain model of
``plain_zokelorn.py``.  Model-level cases run twice: on the host with plain Python standing in for the kernels (what is
under test there is the plan, the parts' wiring, the looped stack's states and caches, the cache manager and the packer), and
on a GPU with the kernels themselves.  Kernel-level cases compare each new kernel with its restatement in ``plain_ops.py`` at
sizes of their own, or with a value that is known by construction."""
import math

import numpy as np
import pytest
import torch

import plain_ops
import plain_zokelorn as plain
import vukavik_util as vu           # the schedule runner and the error measures are not tied to a model
import zokelorn_util as zu


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
    for name, cfg, seed in [("mixed", zu.MIXED, 1), ("tiny", zu.TINY, 2), ("plain", zu.PLAIN, 3), ("serving_heads", zu.SERVING_HEADS, 4)] + \
            [(k, v, 10 + i) for i, (k, v) in enumerate(zu.ONE.items())]:
        out[name] = zu.write_model(str(tmp_path_factory.mktemp(name)), cfg, seed)
        out[name + "/bf16"] = zu.write_model(str(tmp_path_factory.mktemp(name + "bf16")), zu.PLAIN_16 if name == "plain" else cfg, seed, torch.bfloat16,
                                             planted_routes=True)
    return out


_oracles = {}


def _oracle(folder):
    return _oracles.setdefault(folder, zu.Oracle(folder))


def _check(runner, oracle, requests, schedule, dtype):
    got = vu.run_schedule(runner, requests, schedule)
    for rid, toks in requests.items():
        want = oracle.logits(toks)
        e = np.abs(got[rid] - want.numpy()).max(-1) / float(want.max() - want.min())
        zu.within(e, oracle.rounding(toks, dtype), dtype, f"request {rid}", vu.limit(dtype))


def _close(a, b, tol):
    a, b = a.float().cpu(), b.float().cpu()
    assert torch.isfinite(a).all()
    assert float((a - b).abs().max()) <= tol * max(1.0, float(b.abs().max())), f"{float((a - b).abs().max()):.3e}"


# ---- configuration, registry and what a request keeps ---------------------------------------------------------
def test_the_architecture_is_found_by_its_name_and_every_size_comes_from_the_configuration():
    from vapi_b200.config.model import ConfigError, resolve_architecture
    from vapi_b200.parts import FixedDecayMixer, GQAttention, SparseMoE, SwiGLU
    from vapi_b200.parts.base import PagedSpec, StateSpec
    arch = resolve_architecture(zu.MIXED)
    assert arch.name == "Zokelorn"
    plan = arch.plan(arch.parse(zu.MIXED))
    shapes = {s.name: tuple(s.shape) for s in plan.tensor_specs()}
    assert shapes["embed"] == shapes["head"] == (200, 64) and shapes["final.norm"] == shapes["l3.norm1"] == (64,)
    assert shapes["l0.mix.q"] == shapes["l0.mix.k"] == (36, 64) and shapes["l0.mix.v"] == shapes["l0.mix.g"] == (60, 64) and shapes["l0.mix.o"] == (64, 60)
    assert "l0.mix.norm" not in shapes and shapes["l2.mix.norm"] == (5 * 28,), "retention norms without a weight"
    assert shapes["l1.mix.q"] == (80, 64) and shapes["l1.mix.k"] == (40, 64) and shapes["l1.mix.v"] == (24, 64)
    assert shapes["l1.mix.g"] == (4, 64) and shapes["l1.mix.o"] == (64, 48)
    assert shapes["l0.mlp.gate"] == (72, 64) and shapes["l0.mlp.down"] == (64, 72)
    assert shapes["l1.mlp.router"] == (12, 64) and shapes["l1.mlp.e11.up"] == (20, 64) and shapes["l1.mlp.shared.down"] == (64, 28)
    assert shapes["l1.mlp.shared.sg"] == (1, 64) and "l2.mlp.shared.sg" not in shapes and "l2.mlp.shared.up" not in shapes
    assert not any(k.startswith("l3.mlp") for k in shapes) and not any("correction" in k or "norm2" in k for k in shapes)
    # layers 1 to 3 run three times, every pass with a cache or a state of its own
    assert [c.layer for c in plan.order] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4, 5] and all(c.cache_of is None and c.before is None for c in plan.order)
    sites = dict(plan.cache_sites())
    assert set(sites) == set(range(12))
    assert [isinstance(sites[i], PagedSpec) for i in range(12)] == [i in (1, 4, 7, 10) for i in range(12)]
    assert all(s.dtype == torch.float32 and s.shape == (n,) for s, n in ((sites[0], 720), (sites[5], 5 * 8 * 28), (sites[9], 2 * 40 * 16)) if isinstance(s, StateSpec))
    li, re, at = plan.layers[2].mixer, plan.layers[3].mixer, plan.layers[4].mixer
    assert isinstance(li, FixedDecayMixer) and (li.act, li.norm, li.gate, li.qk_scale, li.eps) == ("silu", "all", "sigmoid", 1.0, 1e-5)
    assert (re.act, re.norm, re.gate, re.decay) == (None, "head", "silu", [0.5, 0.995]) and re.qk_scale == pytest.approx(40 ** -0.5)
    assert isinstance(at, GQAttention) and (at.nh, at.nkv, at.d, at.dv, at.chunk, at.rot_dim, at.scale, at.head_gate, at.interleaved) == (3, 1, 16, 36, 37, 16, 0.2, True, True)
    assert isinstance(plan.layers[0].ffn, SwiGLU) and plan.layers[0].ffn.act == "gelu_tanh"
    mo = plan.layers[1].ffn
    assert isinstance(mo, SparseMoE) and (mo.E, mo.top, mo.groups, mo.keep, mo.score, mo.group_top, mo.gate_shared, mo.act) == \
        (12, 3, 3, 2, "sigmoid", 2, True, (0.0, 1.0, 0.0))
    assert len(plan.position_encodings) == 2, "rotary tables are shared only by layers that agree on them"
    free = arch.plan(arch.parse(zu.PLAIN))
    assert [c.layer for c in free.order] == [0, 1, 2, 3, 4] and free.layers[3].mixer.chunk == 0
    for bad in ([{"type": "delta", "mixer": {}, "mlp": None}],
                [zu.layer(zu.attention(heads=3, kv_heads=2))], [zu.layer(zu.attention(dims=22))], [zu.layer(zu.attention(dims=5))],
                [zu.layer(zu.attention(size=0))], [zu.layer(zu.attention(scaling=(0.0, 1.0, 4.0, 8.0)))],
                [zu.layer(zu.memory("retention", decay=[0.5]))],
                [zu.layer({"type": "lightning", "mixer": {"heads": 1, "dim": 4, "vdim": 4}})],
                [zu.layer(zu.attention(), zu.moe(experts=10))], [zu.layer(zu.attention(), zu.moe(groups=(3, 4)))],
                [zu.layer(zu.attention(), zu.moe(top=5, groups=(3, 1)))], [zu.layer(zu.attention(), {"kind": "wide", "ff": 8})]):
        with pytest.raises(ConfigError):
            arch.parse({**zu.MIXED, "layers": bad, "loop": None})
    with pytest.raises(ConfigError):
        arch.parse({**zu.MIXED, "loop": {"start": 2, "stop": 9, "times": 2}})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_are_float32_whatever_the_dtype(dtype, folders, kernels):
    kernels("cpu")
    r = vu.make_runner(folders["tiny"], dtype, "cpu", num_pages=4)
    assert {g.spec.kind: g.tensor.dtype for g in r.cache.state} == {"fixed_decay": torch.float32}
    assert r.plan.layers[0].mixer.powers.shape == (2, 129)


# ---- the plain model itself, by hand ---------------------------------------------------------------------------
def test_the_plain_mechanisms_by_hand():
    f64 = lambda *v: torch.tensor(v, dtype=torch.float64)
    one = lambda *s: torch.ones(s, dtype=torch.float64)
    # frequencies: base 4, four pairs at 1, 1/sqrt 2, ... of wavelengths 2 pi (1, 2^.5, 2, 2^1.5)
    rot = {"dims": 8, "base": 4.0, "scaling": {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 2 * math.pi * 2 ** 0.9}}
    f = plain.frequencies(rot)
    turns = lambda i: 2 ** 0.9 / 2 ** (i / 2)
    s = [(turns(i) - 1.0) / 2.0 for i in range(2)]
    assert f[0] == pytest.approx((1 - s[0]) / 5 + s[0]) and f[1] == pytest.approx(2 ** -0.5 * ((1 - s[1]) / 5 + s[1]))
    assert f[2] == pytest.approx(0.5 / 5) and f[3] == pytest.approx(2 ** -1.5 / 5), "long waves are stretched"
    rot["scaling"]["original"] = 2 * math.pi * 3.5
    assert plain.frequencies(rot)[0] == 1.0, "a short wave stays"
    assert plain.frequencies({"dims": 8, "base": 4.0}) == pytest.approx([1, 2 ** -0.5, 0.5, 2 ** -1.5])
    r = plain.rotate_pairs(f64(1, 2, 3, 4, 5), 3, [1.0, 0.25])
    assert float(r[0]) == pytest.approx(math.cos(3) - 2 * math.sin(3)) and float(r[1]) == pytest.approx(2 * math.cos(3) + math.sin(3))
    assert float(r[2]) == pytest.approx(3 * math.cos(.75) - 4 * math.sin(.75)) and float(r[4]) == 5.0
    # what a position sees: its own chunk up to itself
    assert [plain.visible(i, 3) for i in (0, 2, 3, 7)] == [(0, 0), (0, 2), (3, 3), (6, 7)] and plain.visible(7, None) == (0, 7)
    # equal keys share their weight; the gate halves at a logit of zero; the first token of a chunk sees itself alone
    w = {"q": 0 * one(1, 1), "k": one(1, 1), "v": one(1, 1), "o": one(1, 1), "g": 0 * one(1, 1)}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 2.0, "mask": {"size": 2}}
    out = plain.attention(w, "", m, f64(2.0, 4.0, 10.0)[:, None])
    assert torch.allclose(out[:, 0], f64(1.0, 1.5, 5.0))
    # the recurrence: what was written k steps ago has decayed k times
    o = plain.decayed_memory(one(3, 1, 1), f64(1.0, 0.0, 2.0)[:, None, None], f64(5.0, 7.0, 1.0)[:, None, None], [0.5])
    assert torch.allclose(o.flatten(), f64(5.0, 2.5, 3.25))
    # lightning: silu on all three, one norm over the heads; retention: k / sqrt(dim), a norm per head, a SiLU gate
    si = lambda v: v / (1 + math.exp(-v))
    wl = {"q": one(2, 1), "k": one(2, 1), "v": f64(1.0, -1.0)[:, None], "g": 0 * one(2, 1), "norm": f64(2.0, 3.0), "o": torch.eye(2, dtype=torch.float64)}
    out = plain.lightning(wl, "", {"heads": 2, "dim": 1, "vdim": 1, "decay": [0.5, 0.5]}, f64(1.5)[None], 0.0)
    a, b = si(1.5) ** 3, si(1.5) ** 2 * si(-1.5)
    rms = math.sqrt((a * a + b * b) / 2)
    assert torch.allclose(out[0], f64(a / rms * 2 / 2, b / rms * 3 / 2))
    wr = {"q": one(4, 1), "k": one(4, 1), "v": f64(1.0, -3.0)[:, None], "g": 2 * one(2, 1), "o": torch.eye(2, dtype=torch.float64)}
    out = plain.retention(wr, "", {"heads": 1, "dim": 4, "vdim": 2, "decay": [0.5]}, f64(1.5)[None], 1.0)
    v = f64(1.5, -4.5) * (4 * 1.5 * 1.5 / 2)
    assert torch.allclose(out[0], v / torch.sqrt((v * v).mean() + 1.0) * si(3.0))
    # the router: the group of the two best together wins over the group of the single best
    z = f64(3.0, -4.0, 1.0, 0.9)
    r = {"top": 2, "groups": {"count": 2, "keep": 1}}
    ids, p = plain.choose(z, r)
    sg = lambda v: 1 / (1 + math.exp(-v))
    assert ids == [2, 3] and float(p[0]) == pytest.approx(sg(1.0) / (sg(1.0) + sg(0.9)))
    assert plain.choose(z, {"top": 2})[0] == [0, 2] and plain.choose(z, {"top": 3, "groups": {"count": 4, "keep": 3}})[0] == [0, 2, 3]
    # the tanh form of GELU, not the exact one
    assert float(plain.gelu_tanh(f64(1.3))) == pytest.approx(0.65 * (1 + math.tanh(math.sqrt(2 / math.pi) * (1.3 + 0.044715 * 1.3 ** 3))))
    # a shared expert alone, shut to one half
    wm = {"router": one(1, 1), "e0.gate": 0 * one(1, 1), "e0.up": one(1, 1), "e0.down": one(1, 1), "shared.gate": one(1, 1), "shared.up": one(1, 1),
          "shared.down": one(1, 1), "shared.sg": 0 * one(1, 1)}
    assert float(plain.mixture(wm, "", {"router": {"top": 1}, "shared": {"ff": 1}}, f64(2.0)[None])) == pytest.approx(si(2.0) * 2.0 / 2)
    assert plain.run_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]


def test_the_frequency_rule_of_the_package_is_the_plain_ones():
    from vapi_b200.parts import ScaledRotaryEncoding
    for dims, base, sc in ((12, 30.0, (3.0, 1.0, 5.0, 40.0)), (64, 500000.0, (8.0, 1.0, 4.0, 8192.0)), (2, 7.0, (2.0, 0.5, 0.5, 9.0)), (16, 9.0, (1.0, 1.0, 1.0, 16.0))):
        sc = dict(zip(("factor", "low", "high", "original"), sc))
        f, mult = ScaledRotaryEncoding.frequencies(dims, base, sc)
        assert mult == 1.0 and f == pytest.approx(plain.frequencies({"dims": dims, "base": base, "scaling": sc}), rel=1e-12)


# ---- the model against the plain one: whole prompts, decoding, portions -----------------------------------------
WHOLE = [pytest.param("cpu", "tiny", [19], id="host"),
         pytest.param("cuda", "mixed", [150, 1, 37], marks=pytest.mark.gpu, id="gpu-mixed"),
         pytest.param("cuda", "plain", [70, 2], marks=pytest.mark.gpu, id="gpu-plain"),
         pytest.param("cuda", "serving_heads", [140], marks=pytest.mark.gpu, id="gpu-serving-heads"),
         pytest.param("cuda", "attention", [60], marks=pytest.mark.gpu, id="gpu-attention-alone"),
         pytest.param("cuda", "lightning", [40], marks=pytest.mark.gpu, id="gpu-lightning-alone"),
         pytest.param("cuda", "retention", [40], marks=pytest.mark.gpu, id="gpu-retention-alone"),
         pytest.param("cuda", "experts", [40], marks=pytest.mark.gpu, id="gpu-experts-alone")]


@pytest.mark.parametrize("device,name,lens", WHOLE)
def test_whole_prompt_token_by_token_and_portions_agree_with_the_plain_model(device, name, lens, folders, kernels):
    """Each request alone: its whole prompt in one step; a prompt and then single tokens; portions of changing size
    down to two tokens, cut inside pages and inside chunks."""
    kernels(device)
    oracle = _oracle(folders[name])
    runner = vu.make_runner(folders[name], "float32", device, num_pages=12)
    for i, n in enumerate(lens):
        toks = zu.prompt(oracle.cfg, n, 20 + i)
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
    toks = zu.prompt(oracle.cfg, 170, 5)
    _check(runner, oracle, {"a": toks}, [[("a", 1)]] * 170, "float32")


BATCH = [pytest.param("cpu", "tiny", "float32", [7, 1, 12, 3, 9], 16, id="host"),
         pytest.param("cuda", "mixed", "float32", [70, 1, 33, 150, 2, 64, 17], 16, marks=pytest.mark.gpu, id="gpu-f32"),
         pytest.param("cuda", "mixed/bf16", "bfloat16", [70, 1, 33, 150, 2, 64, 17], 16, marks=pytest.mark.gpu, id="gpu-bf16"),
         pytest.param("cuda", "serving_heads/bf16", "bfloat16", [150, 40, 3, 86, 170], 64, marks=pytest.mark.gpu, id="gpu-bf16-tensor-cores"),
         pytest.param("cuda", "retention/bf16", "bfloat16", [60, 5, 31], 16, marks=pytest.mark.gpu, id="gpu-bf16-retention"),
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
    reqs = {f"r{i}": zu.prompt(oracle.cfg, n, 40 + i) for i, n in enumerate(lens)}
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
            q = min(left[rid], int(torch.tensor([1, 1, 2, 3, 16, 40, 100])[torch.randint(0, 7, (1,), generator=g)]))
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
    """bfloat16: the same request whole, in portions (walked and in chunks), and in a batch with others, against itself."""
    cfg = zu.MIXED if name == "mixed" else zu.SERVING_HEADS
    runner = vu.make_runner(folders[name + "/bf16"], "bfloat16", "cuda", num_pages=12, page_size=64, max_tokens=512)
    toks, other = zu.prompt(cfg, 140, 1), zu.prompt(cfg, 120, 2)
    a = vu.run_schedule(runner, {"a": toks}, [[("a", 140)]])["a"]
    span = float(a.max() - a.min())
    for schedule in ([[("a", q)] for q in vu.cuts(140, [2, 63, 65, 7])], [[("b", 50), ("a", 100)]] + [[("a", 1), ("b", 1)]] * 40 + [[("b", 30)]]):
        reqs = {"a": toks, "b": other} if any(r == "b" for st in schedule for r, _ in st) else {"a": toks}
        b = vu.run_schedule(runner, reqs, schedule)["a"]
        d = np.abs(a - b).max(-1) / span
        assert d.max() < 0.05 and d.mean() < 0.01, f"{d.max():.3e} {d.mean():.3e}"


# ---- faults that random weights would hide ----------------------------------------------------------------------
def _planted_folder(tmp, kind):
    """A model of one layer in which token 1 writes something that only a reader at the right place can see: attention whose
    score for token 1's key stands out, a memory into which nothing but token 1 writes."""
    W, V = 16, 8
    if kind == "attention":
        cfg = zu.config([zu.layer(zu.attention(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, size=24, dims=2, base=1e6, scaling=None))], width=W, vocab=V)
    else:
        cfg = zu.config([zu.layer(zu.memory(kind, heads=1, dim=8, vdim=8, decay=[0.995]))], width=W, vocab=V)
    from vapi_b200.config.model import resolve_architecture
    from vapi_b200.weights import write_random_model
    arch = resolve_architecture(cfg)
    over = {s.name: torch.zeros(s.shape) for s in arch.plan(arch.parse(cfg)).tensor_specs()}
    over["embed"] = torch.zeros(V, W)
    over["embed"][:, 0] = 1.0                 # every token: the reader's mark
    over["embed"][1, 1] = 2.0                 # token 1: the writer's mark
    for k in ("l0.norm1", "final.norm", "l0.mix.norm"):
        if k in over:
            over[k] = torch.ones_like(over[k])
    o = over["l0.mix.o"]
    o[2:10, :8] = torch.eye(8)
    over["head"] = torch.randn(V, W, generator=torch.Generator().manual_seed(5))
    for row in range(over["l0.mix.q"].shape[0] // 8):
        over["l0.mix.q"][8 * row + 5, 0] = 6.0        # (an element that no rotation turns)
    over["l0.mix.k"][5, 1] = 6.0
    over["l0.mix.v"][3, 1] = 4.0
    over["l0.mix.g"][:, 0] = 1.0
    return write_random_model(str(tmp), cfg, 0, overrides=over)


@pytest.mark.parametrize("device,dtype", [pytest.param("cpu", "float32", id="host")] + [pytest.param("cuda", d, marks=pytest.mark.gpu, id=f"gpu-{d}") for d in ("float32", "bfloat16")])
@pytest.mark.parametrize("kind", ["attention", "lightning", "retention"])
def test_one_token_is_seen_exactly_as_long_as_it_should(kind, device, dtype, tmp_path, kernels):
    """Token 1 at one place of a prompt: at a chunk's first and last position, at page borders, at the start.  Attention sees
    it to the end of its chunk of 24 and no further; a memory keeps it, decayed, for good.  In prompts, portions and decoding."""
    kernels(device)
    oracle = zu.Oracle(_planted_folder(tmp_path, kind))
    runner = vu.make_runner(str(tmp_path), dtype, device, num_pages=24)
    n = 60 if device == "cpu" else 150
    for at in ((0, 23, 24) if device == "cpu" else (0, 1, 15, 16, 22, 23, 24, 47, 48, 64, 127, 128)):
        toks = [0] * n
        toks[at] = 1
        want = oracle.logits(toks)
        calm = oracle.logits([0] * n)
        moved = (want - calm).abs().amax(-1)
        seen = [at <= p and (kind != "attention" or p // 24 == at // 24) for p in range(n)]
        assert all((float(m) > 0.05) == s for m, s in zip(moved, seen)), "the plain model itself shows it"
        for schedule in ([[("a", n)]], [[("a", q)] for q in vu.cuts(n, [2, 40, 3, 33])], [[("a", n - 30)]] + [[("a", 1)]] * 30):
            got = vu.run_schedule(runner, {"a": toks}, schedule)["a"]
            off = np.abs(got - want.numpy()).max(-1)
            # (the memories' norms divide what is left of the write by itself: a lost or a kept write shows at full size)
            assert off.max() < (1e-3 if dtype == "float32" else 0.12) * float(want.abs().max()), f"token at {at}: position {off.argmax()} is off by {off.max():.3f}"


# ---- the new kernels against their restatements -------------------------------------------------------------------
#: heads, rows, columns: every split of the rows; sizes that fit no vector access; padding of the chunked form on both sides
STATES = [(3, 1, 3), (2, 7, 5), (5, 12, 20), (3, 24, 40), (2, 32, 64), (2, 48, 24), (3, 64, 72), (2, 128, 128), (1, 100, 8), (2, 200, 136), (1, 256, 64)]


def _memory_case(nh, rows, cols, lens, starts, dtype, seed, extra=8):
    g = torch.Generator().manual_seed(seed)
    n = sum(lens)
    cu, _, pos, slots = zu.step_index(lens, starts, [6, 0, 3, 4, 1][:len(lens)])
    qkv = torch.randn((n, 2 * nh * rows + nh * cols + extra), generator=g).to(dtype)
    state = torch.randn((8, 2, nh * rows * cols + 8), generator=g)
    decay = [1.0, 0.999, 0.7, 0.0, 0.93][:nh]
    return qkv, cu, pos, slots, state, decay


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,rows,cols", STATES)
def test_the_fixed_decay_memory_against_its_restatement(nh, rows, cols, dtype):
    """Single tokens, short and long portions, whole chunks, one token more and less than a chunk, several sequences of which
    some walk and some take chunks; fresh requests over dirty slots and requests that go on; decays of one and of zero; other
    slots and what lies behind the state untouched."""
    from vapi_b200 import ops
    for k, (lens, starts) in enumerate((([1], [0]), ([1, 1, 1], [0, 7, 3]), ([3, 1, 2, 9, 1], [0, 0, 5, 64, 3]), ([31, 32, 33], [0, 5, 0]),
                                        ([127, 128, 129, 1, 40], [0, 9, 2, 100, 0]), ([300], [0]), ([270], [11]))):
        qkv, cu, pos, slots, state, decay = _memory_case(nh, rows, cols, lens, starts, dtype, 100 * rows + cols + k)
        powers = ops.decay_powers(decay, "cuda")
        for act, scale in (("silu", 1.0), (None, rows ** -0.5)):
            want_state, got_state = state.clone(), state.clone().cuda()
            want = plain_ops.fixed_decay_memory(qkv, powers.cpu(), want_state[:, 1], slots, cu, pos, nh, rows, cols, scale, act)
            got = ops.fixed_decay_memory(qkv.cuda(), powers, got_state[:, 1], slots.cuda(), cu.cuda(), pos.cuda(), nh, rows, cols, scale, act,
                                         max_q=max(lens))
            # (bfloat16 inputs are exact in both; SiLU's result is rounded to bfloat16 as an operand, scores and states are not)
            tol = 2e-5 if dtype == torch.float32 else (1e-2 if act else 3e-4)
            _close(got, want, tol)
            _close(got_state, want_state, tol)
            others = [i for i in range(8) if i not in slots.tolist()]
            assert torch.equal(got_state.cpu()[others], state[others]) and torch.equal(got_state.cpu()[:, 0], state[:, 0])
            assert torch.equal(got_state.cpu()[:, 1, nh * rows * cols:], state[:, 1, nh * rows * cols:])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_how_a_sequence_is_cut_changes_its_memory_by_rounding_only(dtype, monkeypatch):
    from vapi_b200 import ops
    nh, rows, cols, n = 3, 40, 24, 400
    g = torch.Generator().manual_seed(2)
    qkv = torch.randn((n, 2 * nh * rows + nh * cols), generator=g).to(dtype).cuda()
    powers = ops.decay_powers([1.0, 0.99, 0.8], "cuda")

    def run(cuts):
        state, outs, at = torch.full((2, nh * rows * cols), 9.0).cuda(), [], 0
        for q in cuts:
            cu, _, pos, slots = (t.cuda() for t in zu.step_index([q], [at], [1]))
            outs.append(ops.fixed_decay_memory(qkv[at:at + q], powers, state, slots, cu, pos, nh, rows, cols, 0.5, None, max_q=q))
            at += q
        return torch.cat(outs), state[1].clone()
    whole = run([n])
    for cuts in ([1] * n, [2, 2, 196, 200], [128, 128, 128, 16], [64, 1, 335], [399, 1]):
        got = run(cuts)
        if dtype == torch.float32:
            assert torch.equal(got[0], whole[0]) and torch.equal(got[1], whole[1]), "the walk does not know where a portion ends"
        else:
            _close(got[0], whole[0], 1e-4)
            _close(got[1], whole[1], 1e-4)
    if dtype == torch.bfloat16:
        monkeypatch.setattr(ops, "FIXED_DECAY_CHUNK_MIN", 0)
        got = run([n])
        _close(got[0], whole[0], 1e-4)
        _close(got[1], whole[1], 1e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_write_is_read_back_from_any_distance(dtype):
    """One token writes, every later one reads: the value times the decay to the distance, at the edges of chunks."""
    from vapi_b200 import ops
    rows, cols, n = 16, 8, 400
    for at in (0, 1, 126, 127, 128, 129, 255, 256, 399):
        for d in (1.0, 0.99, 0.5):
            qkv = torch.zeros((n, 2 * rows + cols))
            qkv[:, 3] = 2.0
            qkv[at, rows + 3] = 1.5
            qkv[:, 2 * rows + 2] = -4.0
            cu, _, pos, slots = (t.cuda() for t in zu.step_index([n], [0], [0]))
            state = torch.full((1, rows * cols), 7.0).cuda()
            out = ops.fixed_decay_memory(qkv.to(dtype).cuda(), ops.decay_powers([d], "cuda"), state, slots, cu, pos, 1, rows, cols, 1.0, None, max_q=n).cpu()
            want = torch.tensor([0.0 if t < at else -12.0 * d ** (t - at) for t in range(n)])
            assert torch.allclose(out[:, 2], want, rtol=5e-5, atol=1e-6), f"written at {at}, decay {d}"
            assert float(out[:, [0, 1, 3, 4, 5, 6, 7]].abs().max()) == 0.0


@pytest.mark.gpu
def test_the_fixed_decay_memory_refuses_what_it_cannot_do():
    from vapi_b200 import ops
    qkv, cu, pos, slots, state, decay = _memory_case(2, 8, 8, [3], [0], torch.float32, 1)
    args = (state.cuda()[:, 1], slots.cuda(), cu.cuda(), pos.cuda())
    with pytest.raises(ops.KernelError):
        ops.fixed_decay_memory(qkv.cuda(), ops.decay_powers([0.5], "cuda"), *args, 2, 8, 8)
    with pytest.raises(ops.KernelError):
        ops.fixed_decay_memory(qkv.cuda(), ops.decay_powers(decay, "cuda"), *args, 2, 8, 8, act="relu")
    with pytest.raises(ops.KernelError):
        ops.fixed_decay_memory(qkv.cuda()[:, :20], ops.decay_powers(decay, "cuda"), *args, 2, 8, 8)
    with pytest.raises(ops.KernelError):
        ops.fixed_decay_memory(qkv, ops.decay_powers(decay, "cpu"), state[:, 1], slots, cu, pos, 2, 8, 8)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_sigmoid_router_with_the_two_best_of_a_group(dtype):
    """Against the restatement (groups of one to eight, all or some kept, with and without the shared expert's gate), and by
    hand: the group of the single best score loses to the group of the two best."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(4)
    for n, W, E, top, groups, keep, gated in ((1, 64, 16, 4, 2, 1, True), (37, 96, 24, 3, 6, 2, True), (70, 66, 8, 2, 8, 3, False), (5, 128, 12, 12, 3, 3, True),
                                              (9, 64, 1, 1, 1, 1, True), (20, 2048, 64, 8, 8, 4, True)):
        h = torch.randn((n, W), generator=g).to(dtype)
        router = torch.randn((E + (1 if gated else 0), W), generator=g) / W ** 0.5
        want_gate = torch.zeros(n) if gated else None
        got_gate = torch.full((n,), 9.0).cuda() if gated else None
        ids, wts, _ = plain_ops.moe_route(h, router, None, E, top, groups, keep, score="sigmoid", group_top=2, shared_gate=want_gate)
        gi, gw, _ = ops.moe_route(h.cuda(), router.cuda(), None, E, top, groups, keep, score="sigmoid", group_top=2, shared_gate=got_gate)
        assert torch.equal(gi.cpu(), ids) and torch.allclose(gw.cpu(), wts, atol=1e-5)
        assert torch.allclose(gw.sum(1).cpu(), torch.ones(n), atol=1e-5)
        if gated:
            assert torch.allclose(got_gate.cpu(), want_gate, atol=1e-5)
    h = torch.zeros((2, 64))
    h[:, 0] = 1.0
    router = torch.zeros((5, 64))
    router[:, 0] = torch.tensor([3.0, -4.0, 1.0, 0.9, -0.5])
    gate = torch.empty(2).cuda()
    ids, wts, _ = ops.moe_route(h.to(dtype).cuda(), router.cuda(), None, 4, 2, 2, 1, score="sigmoid", group_top=2, shared_gate=gate)
    sg = lambda v: 1 / (1 + math.exp(-v))
    assert ids.tolist() == [[2, 3]] * 2 and float(wts[0, 0]) == pytest.approx(sg(1.0) / (sg(1.0) + sg(0.9)), rel=1e-5)
    assert gate.tolist() == pytest.approx([sg(-0.5)] * 2, rel=1e-5)
    ids, _, _ = ops.moe_route(h.to(dtype).cuda(), router[:4].contiguous().cuda(), None, 4, 2, 2, 1, score="sigmoid", group_top=1)
    assert ids.tolist() == [[0, 1]] * 2, "one score a group: the other rule chooses the other group"
    with pytest.raises(ops.KernelError):
        ops.moe_route(h.to(dtype).cuda(), router.cuda(), None, 4, 2, 2, 1, score="tanh")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_beside_a_gated_shared_expert(dtype):
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(6)
    for n, W, ff, E, top in ((1, 64, 24, 6, 2), (90, 96, 40, 8, 3), (300, 64, 10, 3, 3)):
        h, shared = torch.randn((n, W), generator=g).to(dtype), torch.randn((n, W), generator=g).to(dtype)
        router = torch.randn((E + 1, W), generator=g) / W ** 0.5
        up, down = (torch.randn((E, 2 * ff, W), generator=g) * 0.1).to(dtype), (torch.randn((E, W, ff), generator=g) * 0.1).to(dtype)
        gate = torch.empty(n).cuda()
        ids, wts, plan = ops.moe_route(h.cuda(), router.cuda(), None, E, top, 1, 1, score="sigmoid", shared_gate=gate)
        got = ops.moe_experts(h.cuda(), ids, wts, plan, up.cuda(), down.cuda(), shared.cuda(), gated=True, shared_gate=gate)
        want = plain_ops.moe_experts(h, ids.cpu(), wts.cpu(), None, up, down, shared, gated=True, shared_gate=gate.cpu())
        _close(got, want, 2e-5 if dtype == torch.float32 else 2e-2)
        apart = ops.moe_experts(h.cuda(), ids, wts, plan, up.cuda(), down.cuda(), shared.cuda(), gated=True)
        assert float((got - apart).abs().max()) > 0.05, "the gate matters"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_gelu_gate_alone_and_behind_a_product(dtype):
    """Elementwise at widths of every vector form, values from far below zero to far above; then as the epilogue of every
    product that takes it (1 to 16, 17 to 32 and prompt-sized steps) and behind the library's."""
    from vapi_b200 import ops
    g = torch.Generator().manual_seed(7)
    for ff in (1, 6, 12, 40, 328):
        z = torch.randn((9, 2 * ff), generator=g) * 3.0
        z[0, :ff], z[1, :ff], z[2, :ff] = 40.0, -40.0, 0.0
        z = z.to(dtype)
        a, b = z[:, :ff].double(), z[:, ff:].double()
        want = plain.gelu_tanh(a) * b
        _close(ops.swiglu(z.cuda(), act="gelu_tanh"), want, 2e-6 if dtype == torch.float32 else 8e-3)
        assert float((ops.swiglu(z.cuda()).cpu().double() - want).abs().max()) > 0.02, "SiLU is another function"
    for n, K, ff in ((1, 64, 40), (7, 96, 136), (16, 320, 72), (20, 64, 200), (32, 192, 136), (100, 64, 96), (256, 128, 200), (300, 72, 264), (1030, 64, 72)):
        x, w = torch.randn((n, K), generator=g).to(dtype), (torch.randn((2 * ff, K), generator=g) * 0.2).to(dtype)
        y = x.double() @ w.double().t()
        want = plain.gelu_tanh(y[:, :ff]) * y[:, ff:]
        got = ops.linear_swiglu(x.cuda(), w.cuda(), act="gelu_tanh")
        assert got.dtype == dtype and got.shape == (n, ff)
        _close(got, want, 2e-5 if dtype == torch.float32 else 2e-2)
        if dtype == torch.bfloat16 and 16 < n <= 256:
            _close(ops.linear_tc(w.cuda(), act=x.cuda(), epilogue="swiglu", glu="gelu_tanh"), want, 2e-2)
        if dtype == torch.bfloat16 and n > 32:
            _close(ops.prompt_linear(w.cuda(), act=x.cuda(), epilogue="swiglu", glu="gelu_tanh"), want, 2e-2)
    with pytest.raises(ops.KernelError):
        ops.swiglu(z.cuda(), act="gelu")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dk,dv,page", [(20, 12, 8), (64, 64, 64), (128, 128, 64), (48, 48, 16)])
def test_a_planted_key_is_seen_exactly_inside_its_chunk(dtype, dk, dv, page):
    """One key that outweighs all others, at both edges of a chunk, with a gate that halves the output; chunks that are no
    multiple of a page; for single tokens, with split keys, and in portions of every size that picks another kernel."""
    from vapi_b200 import ops
    nh, nkv = 4, 2
    for chunk, klen, j_star, qlen, splits in ((200, 420, 399, 1, 1), (200, 420, 400, 1, 2), (200, 400, 200, 1, 3), (200, 401, 399, 2, 1), (200, 400, 199, 201, 1),
                                              (200, 420, 400, 40, 1), (90, 250, 179, 100, 1), (90, 250, 180, 100, 1), (90, 181, 180, 2, 1), (7, 60, 55, 33, 1),
                                              (7, 60, 56, 3, 1), (1, 9, 5, 9, 1), (64, 130, 127, 66, 1), (64, 130, 128, 66, 1)):
        cache, table, cu, sk = zu.batch([qlen], [klen], page, nkv * (dk + dv), klen + j_star, torch.float32, spread=0.01)
        pg, off = int(table[0, j_star // page]), j_star % page
        for h in range(nkv):
            cache[pg, (h * page + off) * dk] = 10.0
            v0 = nkv * page * dk + (h * page + off) * dv
            cache[pg, v0:v0 + dv] = 1.0
        q = torch.zeros((qlen, nh * dk + nh))
        q[:, :nh * dk:dk] = 2.0                                  # score 20 for the planted key, near zero for the others
        q = q.to(dtype).cuda()
        out = ops.masked_attention(q, q.stride(0), cache.to(dtype).cuda(), page, table.cuda(), cu.cuda(), sk.cuda(), qlen, 1, qlen, klen, nh, nkv, dk, dv,
                                   1.0, chunk=chunk, gate=q[:, nh * dk:], splits=splits).float().cpu()
        for j in range(qlen):
            p = klen - qlen + j
            seen = j_star <= p and j_star // chunk == p // chunk
            assert bool(((out[j] - (0.5 if seen else 0.0)).abs() < 0.03).all()), f"chunks of {chunk}, key {j_star}, query {p}, splits {splits}"


# ---- the engine: scheduler, batching, sampling, entry point -----------------------------------------------------
@pytest.mark.parametrize("device,name,lens,new", [pytest.param("cpu", "tiny", [1, 9, 20], 5, id="host"),
                                                  pytest.param("cuda", "mixed", [1, 33, 80, 7, 64, 40], 10, marks=pytest.mark.gpu, id="gpu")])
def test_greedy_generation_through_the_entry_point(device, name, lens, new, folders, kernels):
    """More requests than slots, prompts cut into portions of 16 beside other requests' decoding; on a GPU pure
    decode steps run as captured graphs, one step ahead of the host.  Slots and pages pass from finished requests to
    waiting ones."""
    kernels(device)
    from vapi_b200 import LLM, SamplingParams
    oracle = _oracle(folders[name])
    llm = LLM(folders[name], dtype="f32", device=device, num_blocks=40, page_size=16, max_concurrent_seqs=4,
              max_batched_tokens=64, prefill_chunk_tokens=16, max_context=256, cuda_graphs=device == "cuda")
    prompts = [zu.prompt(oracle.cfg, n, 50 + i) for i, n in enumerate(lens)]
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
    prompts = [zu.prompt(oracle.cfg, n, 80 + i) for i, n in enumerate([28, 30, 25, 31])]
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
    reqs = {f"r{i}": zu.prompt(cfg, n, 70 + i) for i, n in enumerate([1, 70, 40, 90, 66])}
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
    zu.within(e, slack, dtype, "replay", vu.limit(dtype))
