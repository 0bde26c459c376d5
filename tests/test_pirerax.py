"""The Pirerax decoder in the engine against the plain implementation (tests/plain_pirerax.py): each mechanism's kernels
alone, then whole models of several small shapes through the step function, the scheduler and the replay tool: whole
prompts, token-by-token decoding, portions down to two tokens, unequal batches, slots and pages used again, far keys, page
borders, the first tokens, long decoding and other orders of layers."""
from __future__ import annotations

import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_pirerax as P
from helpers import Replay, assert_close, bf16_noise, random_tokens

F64 = torch.float64
gpu = pytest.mark.gpu


# ----------------------------------------------------------------------------- small shapes
def shape_p1() -> dict:
    """Odd sizes everywhere (a width no tensor-core product takes, a cached row of 26 elements): groups of three query heads,
    a rotation over part of a head, temperatures that change every five tokens, six experts in three groups, a router
    without groups, a layer without feed-forward."""
    return P.make_config(vocab=150, width=100, eps=3e-5, layers=[
        P.latent_layer(3, 10, 6, 14, 20, 0.4, base=300.0, mlp=P.moe(24, 0.8, 6, 3, (3, 2))),
        P.attention_layer(3, 1, 12, 20, 0.5, temp=(0.6, 5)),
        P.parallel_layer((4, 2, 10, 14, 0.45, 6, 70.0), (4, 2, 12, 20, 3), mlp=P.moe(20, 1.5, 5, 2)),
        P.attention_layer(2, 2, 7, 9, 0.6, temp=(-0.2, 16), mlp=P.moe(24, 1.0, 4, 1, (2, 1)))])


def shape_p2() -> dict:
    """Sizes the tensor-core kernels take in bfloat16: value heads narrower and wider than key heads, eight query heads on
    one key head, a rotation over the whole head, many experts of which few are used."""
    return P.make_config(vocab=200, width=128, layers=[
        P.attention_layer(8, 1, 64, 32, 0.2, temp=(0.4, 24), mlp=P.moe(32, 1.0, 12, 3, (4, 2))),
        P.parallel_layer((4, 4, 32, 64, 0.3, 32, 500.0), (4, 1, 16, 32, 4), mlp=P.moe(48, 2.5, 8, 2, (2, 1))),
        P.latent_layer(4, 16, 16, 24, 40, 0.3, base=500.0, mlp=P.moe(64, 0.7, 6, 6, (3, 3)))])


def shape_p3() -> dict:
    """The side-by-side mixer first and last and twice in a row, without a feed-forward behind it (its normed results are
    carried into the next block and into the final norm); a latent of more than 256 values; a convolution of one tap and
    one longer than a page; one head everywhere else."""
    return P.make_config(vocab=90, width=64, eps=1e-4, layers=[
        P.parallel_layer((1, 1, 16, 8, 0.5, 4, 50.0), (1, 1, 8, 8, 1)),
        P.parallel_layer((2, 1, 8, 24, 0.5, 8, 50.0), (3, 3, 16, 8, 9)),
        P.latent_layer(2, 8, 8, 16, 264, 0.5, base=40.0, mlp=P.moe(32, 1.0, 3, 2, (3, 2))),
        P.parallel_layer((2, 2, 40, 16, 0.3, 10, 90.0), (2, 1, 24, 40, 2))])


def shape_p4() -> dict:
    """Twenty heads over one latent, seventeen query heads on one key head (more than a group of the single-token kernel),
    head sizes that need padding, groups of one expert, no rotation in the latent."""
    latent = P.latent_layer(20, 8, 8, 8, 24, 0.5, base=1000.0, mlp=P.moe(16, 1.0, 4, 2, (4, 3)))
    bare = P.latent_layer(2, 24, 0, 16, 32, 0.4, mlp=P.moe(32, 3.0, 2, 1))
    del bare["mixer"]["rot"]
    return P.make_config(vocab=130, width=96, layers=[
        latent, P.attention_layer(17, 1, 24, 40, 0.4, mlp=P.moe(16, 0.5, 8, 4, (2, 2))), bare,
        P.parallel_layer((6, 2, 72, 40, 0.25, 24, 10000.0), (6, 2, 40, 16, 3), mlp=P.moe(48, 1.2, 6, 3, (2, 1)))])


SHAPES = {"p1": (shape_p1, 8), "p2": (shape_p2, 16), "p3": (shape_p3, 8), "p4": (shape_p4, 16)}      # configuration, page size


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """Each shape as it is and with routers that choose every expert, over the same weights."""
    out = {}
    for name, (make, page) in SHAPES.items():
        cfg = make()
        W = P.random_weights(cfg, seed=7 + ord(name[-1]))
        for n, c in ((name, cfg), (name + " all experts", P.all_experts(cfg))):
            out[n] = (P.write_folder(str(tmp_path_factory.mktemp("m")), c, W), c, W, page)
    return out


def pick(folders, name, dtype):
    """Which experts a token goes to is a comparison of scores, and now and then two are so close that bfloat16 rounding of
    the router's input decides otherwise: a different, equally valid computation from there on.  So the bfloat16 runs use
    routers that choose ALL experts (the scores still weigh them, and sorting, segments and sums run as always); the choice
    itself is tested in float32 and on the kernel alone."""
    return folders[name if dtype == "float32" else name + " all experts"]


def engine(folder, dtype, page, tokens=512, batch=256, reqs=4):
    import airun_b200
    return airun_b200.Engine.from_folder(folder, dtype=dtype, page_size=page, cache_tokens=tokens, max_batch_tokens=batch,
                                         max_requests=reqs, max_context=tokens)


def run_schedule(eng, seqs, schedule):
    """schedule: steps, each a list of (request index, tokens to take); wants every token's logits.  Returns
    {request: [T, vocab]} and frees a request when its tokens are used up."""
    from airun_b200 import StepEntry
    at = {i: 0 for i in range(len(seqs))}
    got = {i: [] for i in range(len(seqs))}
    for step in schedule:
        entries = []
        for i, n in step:
            if at[i] == 0:
                eng.manager.add_request(f"q{i}")
            entries.append(StepEntry(f"q{i}", seqs[i][at[i]:at[i] + n], tuple(range(n))))
        out = eng.runner.step(entries).cpu().numpy()
        eng.runner.raise_on_device_error()
        row = 0
        for i, n in step:
            got[i].append(out[row:row + n])
            row += n
            at[i] += n
            if at[i] == len(seqs[i]):
                eng.manager.free_request(f"q{i}")
    eng.manager.check_invariants()
    return {i: np.concatenate(v) for i, v in got.items() if v}


_PLAIN = {}


def plain_logits(cfg, W, seq):
    """The plain logits of a sequence, kept for the next test that asks for the same ones."""
    key = (json.dumps(cfg, sort_keys=True), id(W), tuple(seq))
    if key not in _PLAIN:
        _PLAIN[key] = (P.plain_forward(cfg, W, seq).numpy(), W)                  # W is held, so that its id stays its own
    return _PLAIN[key][0]


def plain_noise(cfg, W, seq):
    """[T, 1]: how far bfloat16 rounding moves each row, the most of five draws: rounding to the nearest, and four times by
    a random amount of up to half a step.  (One draw alone is now and then small by accident on a row that is sensitive:
    a head of the delta rule whose output nearly cancels is blown up by its norm.)"""
    key = (json.dumps(cfg, sort_keys=True), id(W), tuple(seq), "noise")
    if key not in _PLAIN:
        g = torch.Generator().manual_seed(1)
        anywhere = lambda t: t * (1.0 + (torch.rand(t.shape, generator=g, dtype=t.dtype) - 0.5) * 2.0 ** -7)
        draws = [P.plain_forward(cfg, W, seq, rnd=r).numpy() for r in [P.to_bf16_and_back] + [anywhere] * 4]
        exact = plain_logits(cfg, W, seq)
        _PLAIN[key] = (np.max([bf16_noise(d, exact) for d in draws], axis=0), W)
    return _PLAIN[key][0]


def compare(got, cfg, W, seq, dtype, what):
    exact = plain_logits(cfg, W, seq)
    assert_close(got, exact.astype(np.float32), dtype, what, None if dtype == "float32" else plain_noise(cfg, W, seq))


# ----------------------------------------------------------------------------- without a GPU
def test_config_reads_sizes_and_constants():
    from airun_b200.config import PireraxConfig, architecture_name, lookup_architecture
    d = shape_p1()
    assert architecture_name(d) == "Pirerax" and lookup_architecture("Pirerax")[0] is PireraxConfig
    c = PireraxConfig.from_dict(d)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.tie_word_embeddings) == (150, 100, 3e-5, False)
    specs = c.layer_specs()
    assert [s.mixer for s in specs] == ["latent_attention", "softmax_attention", "side_by_side", "softmax_attention"]
    assert [s.feed_forward for s in specs] == ["routed_experts", "", "routed_experts", "routed_experts"]
    assert all(s.arrangement == "pre_norm" for s in specs) and c.ignorable_tensors() == ["l1.norm2"]
    a = specs[0].mixer_args
    assert (a["num_heads"], a["head_dim"], a["rot_dim"], a["value_dim"], a["kv_rank"], a["q_rank"], a["scale"], a["gate"]) == (3, 10, 6, 14, 20, 0, 0.4, "head")
    assert a["position"] == "rotary_neox" and a["position_args"] == dict(rotary_dim=6, theta=300.0) and a["sink"]
    b = specs[1].mixer_args
    assert (b["num_heads"], b["num_kv_heads"], b["key_dim"], b["value_dim"], b["scale"], b["temp_coef"], b["temp_every"]) == (3, 1, 12, 20, 0.5, 0.6, 5)
    assert b["sink"] is True and b["qk_norm"] == "projection" and b["gate"] == "element" and b["position"] == "none"
    p = specs[2].mixer_args
    assert p["combine"] == "norms" and p["norm_eps"] == 3e-5
    assert (p["left"], p["left_args"]["position_args"], p["left_args"]["temp_every"]) == ("softmax_attention", dict(rotary_dim=6, theta=70.0), 0)
    assert "sink" not in p["left_args"] and p["right"] == "gated_delta_rule"
    r = p["right_args"]
    assert (r["num_heads"], r["num_kv_heads"], r["key_dim"], r["value_dim"], r["conv_taps"], r["decay"], r["gate"]) == (4, 2, 12, 20, 3, "head", "silu")
    f = specs[0].ffn_args
    assert (f["num_experts"], f["top"], f["groups"], f["keep_groups"], f["group_best"], f["limit"], f["expert"], f["scores"]) == \
        (6, 3, 3, 2, 2, 0.8, "clamped_glu", "sigmoid")
    assert (specs[2].ffn_args["groups"], specs[2].ffn_args["keep_groups"]) == (1, 1)
    assert PireraxConfig.from_dict(c.to_dict()) == c
    assert PireraxConfig.from_dict(shape_p4()).layer_specs()[2].mixer_args["position"] == "none"


def test_config_lists_every_problem():
    from airun_b200.config import ConfigError, PireraxConfig
    d = P.make_config(vocab=0, width=64, eps=0, layers=shape_p1()["layers"] + [dict(type="other", mixer={}), dict(type="parallel", mixer={})])
    d["layers"][0]["mixer"]["rot"]["dims"] = 8
    d["layers"][0]["mlp"]["router"]["groups"]["count"] = 4
    d["layers"][1]["mixer"]["kv_heads"] = 2
    d["layers"][1]["mixer"]["q_temp"]["every"] = 0
    d["layers"][2]["mixer"]["right"]["conv"] = 0
    d["layers"][2]["mlp"]["expert"]["limit"] = -1
    d["layers"][3]["mlp"]["router"]["top"] = 3
    with pytest.raises(ConfigError) as e:
        PireraxConfig.from_dict(d)
    for piece in ("vocab must be", "norm.eps", "layers[0].mixer.rot.dims must be even and at most 6", "4 groups must divide the 6 experts",
                  "layers[1].mixer.heads (3)", "layers[1].mixer.q_temp.every", "layers[2].mixer.right.conv", "layers[2].mlp.expert.limit",
                  "layers[3].mlp.router.top exceeds", "layers[4] needs", "layers[5].mixer needs 'left' and 'right'"):
        assert piece in str(e.value), piece


def test_declared_tensors_are_the_files_tensors_and_caches_are_owned():
    from airun_b200.config import PireraxConfig
    from airun_b200.engine.model import DecoderModel
    from airun_b200.parts.base import PagedKVSpec, StateSpec
    for name, (make, _) in SHAPES.items():
        m = DecoderModel(PireraxConfig.from_dict(make()), torch.float32, "cpu")
        declared = {s.name: tuple(s.shape) for s in m.weight_specs()}
        shapes = P.tensor_shapes(make())
        assert declared == shapes, (name, set(declared) ^ set(shapes))
        assert m.device_driven()                            # every step can be replayed from a graph
    m = DecoderModel(PireraxConfig.from_dict(shape_p1()), torch.float32, "cpu")
    specs, src = m.cache_specs()
    assert src == [None] * 4 and specs[0] == PagedKVSpec(1, 26, 0, values=False) and specs[1] == PagedKVSpec(1, 12, 0, value_dim=20)
    assert specs[2] == (PagedKVSpec(2, 10, 0, value_dim=14), StateSpec((4 * 12 * 20 + 2 * (2 * 24 + 80),), torch.float32))


def test_plain_mechanisms_against_hand_worked_cases():
    # a sink of ln 3 beside one score of ln 2: the key weighs 2/5; far below every score it weighs nothing
    p = P.plain_softmax_with_sink(torch.tensor([[math.log(2.0), -math.inf]], dtype=F64), torch.tensor(math.log(3.0), dtype=F64))
    assert torch.allclose(p, torch.tensor([[0.4, 0.0]], dtype=F64))
    assert torch.allclose(P.plain_softmax_with_sink(torch.tensor([[0.0, 0.0]], dtype=F64), torch.tensor(-800.0, dtype=F64)), torch.tensor([[0.5, 0.5]], dtype=F64))
    # the temperature steps where p + 1 is a multiple of `every`
    t = P.plain_query_temperature(torch.arange(11), 2.0, 5)
    assert torch.allclose(t, torch.tensor([1.0] * 4 + [1 + 2 * math.log(2.0)] * 5 + [1 + 2 * math.log(3.0)] * 2, dtype=F64))
    # the rotation pairs i with i + dims/2 and leaves the rest
    x = torch.randn(5, 2, 6, dtype=F64)
    r = P.plain_rotate_half(x, torch.arange(5), 4, 100.0)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])
    assert float(r[3, 0, 1]) == pytest.approx(float(x[3, 0, 1] * math.cos(0.3) - x[3, 0, 3] * math.sin(0.3)))
    assert float(r[3, 0, 3]) == pytest.approx(float(x[3, 0, 3] * math.cos(0.3) + x[3, 0, 1] * math.sin(0.3)))
    # routing: the best expert of all lies in a group whose two best sum to less, so it cannot be chosen
    s = torch.tensor([[0.9, 0.1, 0.6, 0.55, 0.2, 0.3]], dtype=F64)
    ids, w = P.plain_route(torch.log(s / (1 - s)), 2, 3, 1)
    assert ids.tolist() == [[2, 3]] and torch.allclose(w, torch.tensor([[0.6, 0.55]], dtype=F64))
    ids, _ = P.plain_route(torch.log(s / (1 - s)), 3, 3, 2)
    assert ids.tolist() == [[0, 2, 3]]
    assert P.plain_route(torch.log(s / (1 - s)), 1, 6, 1)[0].tolist() == [[0]]          # groups of one
    m = P.plain_router_margin(torch.log(s / (1 - s)), 2, 3, 1)
    assert float(m) == pytest.approx(0.15)
    # the gated unit: the gate has no lower clamp
    g, u = torch.tensor([5.0, -30.0, 0.5], dtype=F64), torch.tensor([9.0, -9.0, 0.25], dtype=F64)
    want = [2 / (1 + math.exp(-3.404)) * 3, -30 / (1 + math.exp(1.702 * 30)) * -1, 0.5 / (1 + math.exp(-0.851)) * 1.25]
    assert torch.allclose(P.plain_clamped_unit(g, u, 2.0), torch.tensor(want, dtype=F64))
    # the recurrence: carried across a cut; a unit key with beta 1 replaces what it predicts
    gen = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(12, 2, n, generator=gen, dtype=F64) for n in (3, 3, 4))
    dec, beta = torch.rand(12, 2, generator=gen, dtype=F64), torch.rand(12, 2, generator=gen, dtype=F64)
    o, S = P.plain_delta_recurrence(q, k, v, dec, beta)
    o1, S1 = P.plain_delta_recurrence(q[:5], k[:5], v[:5], dec[:5], beta[:5])
    o2, S2 = P.plain_delta_recurrence(q[5:], k[5:], v[5:], dec[5:], beta[5:], state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
    kk = torch.zeros(12, 2, 3, dtype=F64)
    kk[..., 1] = 1.0
    assert torch.allclose(P.plain_delta_recurrence(kk, kk, v, dec, torch.ones(12, 2, dtype=F64))[0], v)
    # the convolution's last tap is the token's own
    y = P.plain_short_conv(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[3.0, 5.0]]))
    assert y.flatten().tolist() == [5.0, 53.0, 530.0]


# ----------------------------------------------------------------------------- kernels alone
def dev(t, dtype=torch.float32):
    return t.to("cuda", dtype).contiguous()


def batch_ctx(spans, slots=None):
    """The device arrays of a step whose request r brings rows spans[r] = (first position, end)."""
    from airun_b200.engine.batch import Workspace
    lens = [b - a for a, b in spans]
    cu = torch.tensor(np.cumsum([0] + lens), dtype=torch.int32, device="cuda")
    req = torch.cat([torch.full((n,), r) for r, n in enumerate(lens)]).to("cuda", torch.int32)
    pos = torch.cat([torch.arange(a, b) for a, b in spans]).to("cuda", torch.int32)
    ends = torch.tensor([b for _, b in spans], dtype=torch.int32, device="cuda")
    return SimpleNamespace(req_of_token=req, cu_tokens=cu, positions=pos, context_lens=ends, num_reqs=len(spans),
                           num_tokens=sum(lens), decode_only=all(n == 1 for n in lens), query_lens=lens,
                           context_lens_host=[b for _, b in spans], max_query_len=max(lens), max_context_len=max(b for _, b in spans),
                           ws=Workspace(torch.device("cuda"), 8 << 20), ws_main=Workspace(torch.device("cuda"), 8 << 20), extras={},
                           state_slots=torch.tensor(slots if slots is not None else list(range(len(spans))), dtype=torch.int32, device="cuda"),
                           err=torch.zeros(1, dtype=torch.int32, device="cuda"))


def scrambled_table(seq_lens, page, g):
    """(block table int32 [requests, blocks], pages of the pool): pages handed out in a random order."""
    blocks = [(n + page - 1) // page for n in seq_lens]
    num_pages = sum(blocks) + 3
    perm = torch.randperm(num_pages, generator=g).tolist()
    bt = torch.full((len(seq_lens), max(blocks)), -1, dtype=torch.int32)
    for r, nb in enumerate(blocks):
        for blk in range(nb):
            bt[r, blk] = perm.pop()
    return bt.cuda(), num_pages


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,n", [(5, 100), (1, 48), (90, 328), (3, 2051), (70, 2048), (2, 4096), (66, 9001), (3, 20000)])
def test_two_normed_results_join_in_one_pass(T, n, dtype):
    from airun_b200.kernels import ops
    from airun_b200.parts.base import PostNormWrite
    g = torch.Generator().manual_seed(T + n)
    x, y, z = 3 * torch.randn(T, n, generator=g), torch.randn(T, n, generator=g) * torch.rand(T, 1, generator=g), 40 * torch.randn(T, n, generator=g)
    a, c, b = (1 + 0.3 * torch.randn(n, generator=g) for _ in range(3))
    v = x.double() + 0.5 * (P.plain_rmsnorm(y.double(), a.double(), 1e-4) + P.plain_rmsnorm(z.double(), c.double(), 1e-4))
    h = P.plain_rmsnorm(v, b.double(), 1e-3)
    write = PostNormWrite(dev(y), dev(a), 1e-4, dev(z), dev(c), 0.5).norm_args()
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    xd, out = dev(x), torch.empty(T, n, device="cuda", dtype=dtype)
    ops.sandwich_norm(xd, out, w_pre=dev(b), eps_pre=1e-3, **write)
    assert torch.allclose(xd.cpu().double(), v, rtol=3e-6, atol=3e-6) and torch.allclose(out.cpu().double(), h, rtol=tol, atol=tol)
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device="cuda")          # chosen rows: x stays as it is
    xd, few = dev(x), torch.empty(3, n, device="cuda", dtype=dtype)
    ops.sandwich_norm(xd, few, w_pre=dev(b), eps_pre=1e-3, rows=rows, **write)
    assert torch.equal(xd.cpu(), x) and torch.allclose(few.cpu().double(), h[rows.long().cpu()], rtol=tol, atol=tol)
    ops.sandwich_norm(xd, None, **write)                                               # the norms and the add alone
    assert torch.allclose(xd.cpu().double(), v, rtol=3e-6, atol=3e-6)


# ---- grouped attention: one norm over all heads, rotation or temperature, gate per element
def attention_case(seq_lens, new_lens, nh, nkv, D, Dv, page, dtype, seed, rot=None, temp=(0.0, 0), spike=None, norm=True):
    """Keys and values written through the prologue kernel for the first len - new tokens of every request, then the last
    ``new`` tokens of each as one batch; the projections' last nh * Dv columns are the gate's.  Returns the projections, the
    norm weights, the cache, the last batch's (spans, ctx, live requests), its q and its projections on the device."""
    from airun_b200.kernels import ops
    from airun_b200.parts.base import make_part
    g = torch.Generator().manual_seed(seed)
    width = nh * D + nkv * (D + Dv) + nh * Dv
    reqs = []
    for n in seq_lens:
        proj = torch.randn(n, width, generator=g) * (0.5 + torch.rand(n, 1, generator=g))
        if spike is not None:
            spike(proj, n)
        reqs.append(proj)
    qw, kw = (1.5 + 0.3 * torch.randn(nh * D, generator=g), 1.5 + 0.3 * torch.randn(nkv * D, generator=g)) if norm else (None, None)
    kind, r, inv = ops.ROPE_NONE, 0, None
    if rot:
        kind, r, inv = make_part("position", "rotary_neox", rotary_dim=rot[0], theta=rot[1], device="cuda").fused()
    bt, num_pages = scrambled_table(seq_lens, page, g)
    cache = SimpleNamespace(pool=torch.zeros(num_pages, nkv * page * (D + Dv), device="cuda", dtype=dtype), block_table=bt, page_size=page, shared=False)
    last = None
    for phase in (0, 1):
        spans = [(0, n - m) if phase == 0 else (n - m, n) for n, m in zip(seq_lens, new_lens)]
        live = [(i, s) for i, s in enumerate(spans) if s[1] > s[0]]
        if not live:
            continue
        ctx = batch_ctx([s for _, s in live])
        cache.block_table = bt[[i for i, _ in live]].contiguous()
        proj = dev(torch.cat([reqs[i][a:e] for i, (a, e) in live]))
        q = torch.empty(proj.shape[0], nh * D, device="cuda", dtype=dtype)
        ops.qkv_prepare(proj, None, None if qw is None else dev(qw), None if kw is None else dev(kw), False, 1e-5, kind, r, inv, temp[0], temp[1],
                        q, cache, ctx, nh, nkv, D, Dv, store=True, whole_norm=norm)
        assert int(ctx.err.item()) == 0
        last = ([s for _, s in live], ctx, [i for i, _ in live], q, proj)
    return reqs, (qw, kw), cache, last


def plain_qkv(proj, weights, nh, nkv, D, Dv, rot, temp):
    n, p = proj.shape[0], proj.double()
    q, k, v = p[:, :nh * D], p[:, nh * D:(nh + nkv) * D], p[:, (nh + nkv) * D:(nh + nkv) * D + nkv * Dv].reshape(n, nkv, Dv)
    if weights[0] is not None:
        q, k = P.plain_rmsnorm(q, weights[0].double(), 1e-5), P.plain_rmsnorm(k, weights[1].double(), 1e-5)
    q, k = q.reshape(n, nh, D), k.reshape(n, nkv, D)
    pos = torch.arange(n)
    if rot:
        q, k = P.plain_rotate_half(q, pos, *rot), P.plain_rotate_half(k, pos, *rot)
    if temp[1]:
        q = q * P.plain_query_temperature(pos, *temp)[:, None, None]
    return q, k, v


def plain_case(reqs, weights, spans, live, nh, nkv, D, Dv, scale, rot, temp, sink, gated):
    outs = []
    for i, (a, e) in zip(live, spans):
        q, k, v = plain_qkv(reqs[i][:e], weights, nh, nkv, D, Dv, rot, temp)
        vis = P.plain_causal(e)
        o = torch.zeros(e, nh, Dv, dtype=F64)
        for h in range(nh):
            kv = h // (nh // nkv)
            s = (q[:, h] @ k[:, kv].T * scale).masked_fill(~vis, -math.inf)
            o[:, h] = P.plain_softmax_with_sink(s, None if sink is None else sink[h].double()) @ v[:, kv]
        o = o.reshape(e, nh * Dv)
        if gated:
            o = o * torch.sigmoid(reqs[i][:e, -nh * Dv:].double())
        outs.append(o[a:e])
    return torch.cat(outs)


def run_attention(case, nh, nkv, D, Dv, scale, sink, gated, tensor_cores=False):
    from airun_b200.kernels import fast, ops
    _, _, cache, (spans, ctx, live, q, proj) = case
    gate = proj[:, proj.shape[1] - nh * Dv:] if gated else None
    sd = None if sink is None else dev(sink)
    wide = torch.zeros(q.shape[0], nh * Dv + 16, device="cuda", dtype=q.dtype)
    out = wide[:, 8:8 + nh * Dv]
    if tensor_cores:
        part = SimpleNamespace(D=D, Dv=Dv, nh=nh, nkv=nkv, scale=scale, table=None, sink=sd, window=0, out_scale=1.0, tail=-1)
        assert fast.softmax_attention_bf16(ctx, q, out, cache, part, gate)
    else:
        ops.softmax_attention(q, out, cache, ctx, nh, nkv, D, Dv, scale, None, sd, 0, 1.0, gate=gate)
    assert int(ctx.err.item()) == 0 and float(wide[:, :8].abs().max()) == 0 and float(wide[:, 8 + nh * Dv:].abs().max()) == 0
    return out.float().cpu().double()


ATT_SHAPES = [  # heads, kv heads, D, Dv, rotation, temperature, page
    (3, 1, 12, 20, (6, 300.0), (0.0, 0), 8), (4, 2, 88, 72, None, (0.6, 5), 16), (8, 8, 32, 64, (32, 500.0), (0.0, 0), 16),
    (2, 1, 130, 6, (10, 90.0), (0.3, 7), 8), (6, 2, 64, 128, (24, 500.0), (0.0, 0), 32), (17, 1, 24, 40, None, (-0.2, 16), 8),
    (16, 1, 16, 8, None, (0.0, 0), 8), (2, 2, 256, 200, (256, 500.0), (0.0, 0), 8), (5, 1, 7, 9, (4, 40.0), (0.5, 3), 24)]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", ATT_SHAPES)
def test_norm_over_the_whole_projection_and_gated_attention(shape, dtype):
    """A portion beside a whole prompt beside a single token over scrambled pages; q and the cached rows themselves; with
    and without sink and gate."""
    nh, nkv, D, Dv, rot, temp, page = shape
    seqs, new = [70, 23, 91], [13, 23, 1]
    case = attention_case(seqs, new, nh, nkv, D, Dv, page, dtype, 5, rot, temp)
    reqs, weights, cache, (spans, ctx, live, q, proj) = case
    tol = 2e-5 if dtype == torch.float32 else 5e-2
    for j, i in enumerate(live):
        qp, kp, vp = plain_qkv(reqs[i], weights, nh, nkv, D, Dv, rot, temp)
        for pos in (0, 7, 8, seqs[i] - 1):
            flat = cache.pool[int(cache.block_table[j, pos // page])].double().cpu()
            kr, vr = flat[:nkv * page * D].view(nkv, page, D)[:, pos % page], flat[nkv * page * D:].view(nkv, page, Dv)[:, pos % page]
            assert torch.allclose(kr, kp[pos], atol=tol, rtol=tol) and torch.allclose(vr, vp[pos], atol=tol, rtol=tol)
        a, e = spans[j]
        rows = q[int(ctx.cu_tokens[j]):int(ctx.cu_tokens[j + 1])].double().cpu().view(e - a, nh, D)
        assert torch.allclose(rows, qp[a:e], atol=tol, rtol=tol)
    scale = 0.7 * D ** -0.5
    sink = 1.0 + torch.randn(nh, generator=torch.Generator().manual_seed(2))
    for s, gated in ((sink, True), (None, True), (sink, False)):
        got = run_attention(case, nh, nkv, D, Dv, scale, s, gated)
        want = plain_case(reqs, weights, spans, live, nh, nkv, D, Dv, scale, rot, temp, s, gated)
        assert torch.allclose(got, want, atol=tol, rtol=tol), float((got - want).abs().max())


@gpu
@pytest.mark.parametrize("shape", [s for s in ATT_SHAPES if s[2] <= 128 and s[3] <= 128])
@pytest.mark.parametrize("new", [[13, 23, 1], [1, 1, 1], [130, 70, 64]])
def test_gated_attention_on_the_tensor_cores(shape, new):
    """A portion beside a whole prompt beside a single token; single tokens alone (700, 23 and 1500 keys, cut into slices,
    some of them empty); several tiles of several requests; against the plain kernel and the formula."""
    nh, nkv, D, Dv, rot, temp, page = shape
    seqs = [70, 23, 91] if new == [13, 23, 1] else [700, 23, 1500] if new[0] == 1 else [300, 70, 65]
    case = attention_case(seqs, new, nh, nkv, D, Dv, page, torch.bfloat16, 6, rot, temp)
    reqs, weights, cache, (spans, ctx, live, q, proj) = case
    scale, sink = 0.7 * D ** -0.5, 1.0 + torch.randn(nh, generator=torch.Generator().manual_seed(2))
    for s in (sink, None):
        want = plain_case(reqs, weights, spans, live, nh, nkv, D, Dv, scale, rot, temp, s, True)
        got = run_attention(case, nh, nkv, D, Dv, scale, s, True, tensor_cores=True)
        plain = run_attention(case, nh, nkv, D, Dv, scale, s, True)
        assert torch.allclose(got, want, atol=1e-1, rtol=3e-2), float((got - want).abs().max())        # bfloat16 q and rows against float64
        assert torch.allclose(got, plain, atol=2e-2, rtol=2e-2), float((got - plain).abs().max())      # the same inputs: only the weights' rounding


@gpu
@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("key_at", [0, 7, 8, 299, 444, 599])
@pytest.mark.parametrize("new", [1, 2, 40])
def test_one_key_that_stands_out(key_at, new, tensor_cores):
    """Among 600 keys ONE has a large score with the last query; its value, times the gate, must be what the query returns:
    far back, at position 0, at a page border, and the token itself; a sink far below it takes nothing, one far above takes all."""
    n, nh, nkv, D, Dv, page = 600, 2, 1, 32, 24, 8

    def spike(proj, n_):
        proj *= 0.05
        proj[n_ - 1, 20:nh * D:D] = 6.0                     # the last token's query heads point along dimension 20
        proj[key_at, nh * D + 20] = 6.0                     # and so does the key at key_at
        proj[key_at, nh * D + D:nh * D + D + Dv] = torch.linspace(-2, 2, Dv)
    case = attention_case([n], [new], nh, nkv, D, Dv, page, torch.bfloat16 if tensor_cores else torch.float32, 3, spike=spike, norm=False)
    reqs, weights, cache, (spans, ctx, live, q, proj) = case
    sink = torch.tensor([-20.0, 90.0])
    got = run_attention(case, nh, nkv, D, Dv, 1.0, sink, True, tensor_cores)
    gate = torch.sigmoid(reqs[0][n - 1, -nh * Dv:].double())
    assert torch.allclose(got[-1, :Dv], torch.linspace(-2, 2, Dv).double() * gate[:Dv], atol=2e-2 if tensor_cores else 1e-3)
    assert float(got[-1, Dv:].abs().max()) < 1e-6
    want = plain_case(reqs, weights, spans, live, nh, nkv, D, Dv, 1.0, None, (0.0, 0), sink, True)
    assert torch.allclose(got, want, atol=3e-2 if tensor_cores else 2e-5, rtol=3e-2 if tensor_cores else 1e-5)


# ---- attention over a latent with direct queries, rotated pairs (i, i + r/2), a gate per head
def latent_case(seq_lens, new_lens, H, D, R, rd, page, dtype, seed, rot=None, spike=None):
    """Rows [queries H * (D + rd) | latent R | rotated key rd | gates H] through the prologue kernel, as attention_case.  The
    unrotated queries are carried into the latent space by a fixed matrix per head (as the engine's per-head product does)."""
    from airun_b200.kernels import ops
    from airun_b200.parts.base import make_part
    from airun_b200.parts.latent_attention import head_linear
    g = torch.Generator().manual_seed(seed)
    uk = P.to_bf16_and_back(torch.randn(H, D, R, generator=g) / math.sqrt(R))
    wkv = 1 + 0.3 * torch.randn(R, generator=g)
    reqs = []
    for n in seq_lens:
        rows = torch.randn(n, H * (D + rd) + R + rd + H, generator=g)
        if spike is not None:
            spike(rows, n, uk, wkv)
        reqs.append(rows)
    inv = make_part("position", "rotary_neox", rotary_dim=rot[0], theta=rot[1], device="cuda").inv_freq if rot else None
    bt, num_pages = scrambled_table(seq_lens, page, g)
    cache = SimpleNamespace(pool=torch.zeros(num_pages, page * (R + rd), device="cuda", dtype=dtype), block_table=bt, page_size=page, shared=False)
    last = None
    for phase in (0, 1):
        spans = [(0, n - m) if phase == 0 else (n - m, n) for n, m in zip(seq_lens, new_lens)]
        live = [(i, s) for i, s in enumerate(spans) if s[1] > s[0]]
        if not live:
            continue
        ctx = batch_ctx([s for _, s in live])
        cache.block_table = bt[[i for i, _ in live]].contiguous()
        rows = dev(torch.cat([reqs[i][a:e] for i, (a, e) in live]))
        T = rows.shape[0]
        qn, qlat = torch.empty(T, H * D, device="cuda", dtype=dtype), torch.zeros(T, H * (R + rd), device="cuda", dtype=dtype)
        ops.latent_query(rows, qn, qlat, H, D, R, rd, rot[0] if rot else 0, inv, 1.0, ctx, rope_kind=ops.ROPE_NEOX, wkv=dev(wkv), eps=1e-5, cache=cache)
        head_linear(ctx, qn.view(T, H, D), dev(uk.transpose(1, 2), dtype), qlat.view(T, H, R + rd)[:, :, :R])
        assert int(ctx.err.item()) == 0
        last = ([s for _, s in live], ctx, [i for i, _ in live], qlat, rows[:, rows.shape[1] - H:])
    return reqs, uk, wkv, cache, last


def plain_latent(rows, uk, wkv, H, D, R, rd, scale, rot, sink, gated, window=0):
    n, r = rows.shape[0], rows.double()
    q, c, kr = r[:, :H * (D + rd)].reshape(n, H, D + rd), r[:, H * (D + rd):H * (D + rd) + R], r[:, H * (D + rd) + R:H * (D + rd) + R + rd]
    c, kr, qr = P.plain_rmsnorm(c, wkv.double(), 1e-5), kr[:, None], q[..., D:]
    if rot:
        kr, qr = P.plain_rotate_half(kr, torch.arange(n), *rot), P.plain_rotate_half(qr, torch.arange(n), *rot)
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    vis = (d >= 0) & ((d < window) if window else True)
    out = torch.zeros(n, H, R, dtype=F64)
    for h in range(H):
        s = (q[:, h, :D] @ (c @ uk[h].double().T).T + qr[:, h] @ kr[:, 0].T) * scale
        out[:, h] = P.plain_softmax_with_sink(s.masked_fill(~vis, -math.inf), None if sink is None else sink[h].double()) @ c
    if gated:
        out = out * torch.sigmoid(r[:, -H:])[:, :, None]
    return out.reshape(n, H * R), c, kr[:, 0], qr


def run_latent(case, H, R, rd, scale, sink, gated, window=0, tensor_cores=False):
    from airun_b200.kernels import fast, ops
    cache, (spans, ctx, live, qlat, gate) = case[3], case[4]
    out = torch.zeros(qlat.shape[0], H * R, device="cuda", dtype=qlat.dtype)
    sd = None if sink is None else dev(sink)
    if tensor_cores:
        part = SimpleNamespace(nh=H, R=R, rd=rd, scale=scale, window=window, sink=sd)
        assert fast.latent_attention_bf16(ctx, qlat, out, cache, part, gate if gated else None)
    else:
        ops.latent_attention(qlat, out, cache, ctx, H, R, rd, scale, window, sd, gate if gated else None)
    assert int(ctx.err.item()) == 0
    return out.float().cpu().double()


LATENT_SHAPES = [  # heads, D, R, rd, rotation, page
    (3, 10, 20, 6, (6, 300.0), 8), (2, 16, 64, 16, (16, 500.0), 16), (1, 5, 130, 7, (4, 90.0), 24), (4, 16, 16, 0, None, 8),
    (20, 8, 24, 8, (8, 1000.0), 8), (16, 32, 264, 40, (40, 10000.0), 16), (33, 16, 512, 64, (64, 10000.0), 16), (2, 16, 600, 40, (40, 50.0), 16)]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_direct_latent_queries_and_gated_heads(shape, dtype):
    """Queries, cached rows and the plain attention over scrambled pages: a portion, a whole prompt and a single token."""
    H, D, R, rd, rot, page = shape
    seqs, new = [70, 9, 33], [13, 9, 1]
    case = latent_case(seqs, new, H, D, R, rd, page, dtype, H + R, rot)
    reqs, uk, wkv, cache, (spans, ctx, live, qlat, gate) = case
    tol = 3e-5 if dtype == torch.float32 else 5e-2
    scale, sink = 0.8 * (D + rd) ** -0.5, 1.0 + torch.randn(H, generator=torch.Generator().manual_seed(3))
    want = []
    for j, i in enumerate(live):
        a, e = spans[j]
        o, c, kr, qr = plain_latent(reqs[i][:e], uk, wkv, H, D, R, rd, scale, rot, sink, True)
        want.append(o[a:e])
        for pos in (0, 7, 8, e - 1):
            row = cache.pool[int(cache.block_table[j, pos // page])].view(page, R + rd)[pos % page].double().cpu()
            assert torch.allclose(row[:R], c[pos], atol=tol, rtol=tol) and torch.allclose(row[R:], kr[pos], atol=tol, rtol=tol)
        got_q = qlat[int(ctx.cu_tokens[j]):int(ctx.cu_tokens[j + 1])].view(e - a, H, R + rd)[:, :, R:].double().cpu()
        assert torch.allclose(got_q, qr[a:e], atol=tol, rtol=tol)
    got = run_latent(case, H, R, rd, scale, sink, True)
    assert torch.allclose(got, torch.cat(want), atol=tol, rtol=tol), float((got - torch.cat(want)).abs().max())


@gpu
@pytest.mark.parametrize("window", [0, 37])
@pytest.mark.parametrize("new", [[13, 23, 1], [1, 1, 1], [130, 70, 64], [2, 1, 300]])
@pytest.mark.parametrize("shape", [s for s in LATENT_SHAPES if (s[2] + s[3]) % 8 == 0])
def test_gated_latent_attention_on_the_tensor_cores(shape, new, window):
    """Portions beside single tokens; single tokens alone (700, 23 and 1500 keys, cut into slices, some of them empty);
    several tiles of several requests; head counts above and below a row tile, more than 256 output columns."""
    H, D, R, rd, rot, page = shape
    seqs = [700, 23, 1500] if new == [1, 1, 1] else [n + 57 * i for i, n in enumerate((150, 70, 200))]
    case = latent_case(seqs, new, H, D, R, rd, page, torch.bfloat16, H + R, rot)
    reqs, uk, wkv, cache, (spans, ctx, live, qlat, gate) = case
    scale, sink = 0.8 * (D + rd) ** -0.5, 1.0 + torch.randn(H, generator=torch.Generator().manual_seed(3))
    for gated, s in ((True, sink), (False, None)):
        got = run_latent(case, H, R, rd, scale, s, gated, window, tensor_cores=True)
        plain = run_latent(case, H, R, rd, scale, s, gated, window)
        assert torch.allclose(got, plain, atol=3e-2, rtol=3e-2), float((got - plain).abs().max())
    want = torch.cat([plain_latent(reqs[i][:e], uk, wkv, H, D, R, rd, scale, rot, None, False, window)[0][a:e] for i, (a, e) in zip(live, spans)])
    assert torch.allclose(got, want, atol=1e-1, rtol=5e-2), float((got - want).abs().max())


@gpu
@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("key_at", [0, 7, 8, 63, 64, 299, 444, 599])
@pytest.mark.parametrize("new", [1, 2, 40])
def test_one_latent_that_stands_out(key_at, new, tensor_cores):
    """The last query points along ONE cached latent: far back, the first token, at a page's and a key tile's border, the
    token itself; the result is that latent times the head's gate."""
    H, D, R, rd, page, n = 2, 32, 32, 8, 8, 600

    def spike(rows, n_, uk, wkv):
        uk.copy_(torch.eye(D, R).expand(H, D, R))           # latent space and query space are the same
        rows[:, H * (D + rd) + R:H * (D + rd) + R + rd] = 0.0
        c = P.plain_rmsnorm(rows[key_at, H * (D + rd):H * (D + rd) + R].double(), wkv.double(), 1e-5)
        for h in range(H):
            rows[n_ - 1, h * (D + rd):h * (D + rd) + D] = (4.0 * c / c.norm() * (4 if h == 0 else 0)).float()
    case = latent_case([n], [new], H, D, R, rd, page, torch.bfloat16 if tensor_cores else torch.float32, 11, (8, 100.0), spike)
    reqs, uk, wkv, cache, (spans, ctx, live, qlat, gate) = case
    sink = torch.tensor([-20.0, 60.0])
    got = run_latent(case, H, R, rd, 1.0, sink, True, tensor_cores=tensor_cores)
    want, c, _, _ = plain_latent(reqs[0], uk, wkv, H, D, R, rd, 1.0, (8, 100.0), sink, True)
    tol = 3e-2 if tensor_cores else 1e-4
    assert torch.allclose(got, want[n - new:], atol=tol, rtol=tol), float((got - want[n - new:]).abs().max())
    gate0 = float(torch.sigmoid(reqs[0][n - 1, -H].double()))
    assert torch.allclose(got[-1, :R], c[key_at] * gate0, atol=8e-2) and float(got[-1, R:].abs().max()) < 1e-6


@gpu
@pytest.mark.parametrize("T", [1, 5, 64, 129, 300])
@pytest.mark.parametrize("heads,K,N,pad_x,pad_out", [(3, 24, 40, 0, 0), (16, 128, 512, 0, 64), (5, 72, 300, 8, 3), (1, 64, 16, 0, 0), (20, 8, 264, 16, 8), (2, 520, 24, 0, 0)])
def test_products_per_head_in_one_launch(heads, K, N, pad_x, pad_out, T):
    """Column slices of wider rows on both sides; what lies between the slices (set to large numbers) does not show, nor is
    anything written there."""
    from airun_b200.kernels import fast
    g = torch.Generator().manual_seed(K + N)
    x = torch.full((T, heads, K + pad_x), 1e4)
    x[:, :, :K] = P.to_bf16_and_back(torch.randn(T, heads, K, generator=g))
    w = P.to_bf16_and_back(torch.randn(heads, N, K, generator=g) / math.sqrt(K))
    xd, out = dev(x, torch.bfloat16), torch.full((T, heads, N + pad_out), 7.0, device="cuda", dtype=torch.bfloat16)
    ctx = batch_ctx([(0, T)])
    assert fast.head_linear_bf16(ctx, xd[:, :, :K], dev(w, torch.bfloat16), out[:, :, :N])
    want = torch.einsum("thk,hnk->thn", x[:, :, :K].double(), w.double())
    assert int(ctx.err.item()) == 0 and torch.allclose(out[:, :, :N].cpu().double(), want, atol=2e-2, rtol=1e-2)
    assert (out[:, :, N:] == 7.0).all()


# ---- routed experts
@gpu
@pytest.mark.parametrize("n_out,top,groups,keep", [(6, 3, 3, 2), (20, 4, 2, 1), (9, 3, 3, 2), (5, 5, 5, 5), (4, 1, 4, 1), (40, 6, 1, 1), (64, 8, 8, 4), (12, 2, 4, 3)])
def test_group_routing_by_sigmoid_scores(n_out, top, groups, keep):
    from airun_b200.kernels import ops
    g = torch.Generator().manual_seed(n_out)
    T = 77
    z = 2 * torch.randn(T, n_out + 3, generator=g)
    z[3] = 20 + z[3]                                         # scores that all round to 1: still ranked
    ids, rank = (torch.empty(T, top, dtype=torch.int32, device="cuda") for _ in range(2))
    wts = torch.empty(T, top, device="cuda")
    counts, seg = torch.zeros(n_out, dtype=torch.int32, device="cuda"), torch.empty(n_out + 1, dtype=torch.int32, device="cuda")
    req = torch.zeros(T, dtype=torch.int32, device="cuda")
    req[5] = -1
    ops.moe_route_grouped(dev(z)[:, :n_out], n_out, top, groups, keep, 1.0, None, req, ids, wts, rank, counts, seg, sigmoid_scores=True,
                          group_best=2, renorm=False)
    want_ids, want_w = P.plain_route(z[:, :n_out].double(), top, groups, keep)
    ids, wts, rank = ids.cpu(), wts.cpu(), rank.cpu()
    rows = [t for t in range(T) if t != 5 and not (t == 3 and keep < groups)]        # (float32 sums of saturated groups may tie)
    assert ids[5].tolist() == [-1] * top
    assert torch.equal(ids[rows].long(), want_ids[rows])
    assert torch.allclose(wts[rows].double(), want_w[rows], atol=1e-6, rtol=1e-5)
    real = [t for t in range(T) if t != 5]
    for e in range(n_out):
        mine = sorted(int(rank[t, k]) for t in real for k in range(top) if int(ids[t, k]) == e)
        assert mine == list(range(len(mine))) and int(counts[e]) == len(mine)
    assert seg.cpu().tolist() == np.cumsum([0] + counts.cpu().tolist()).tolist()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,I,E,top,groups,limit", [(33, 100, 24, 6, 3, (3, 2), 0.5), (200, 128, 64, 8, 2, (4, 2), 1.0), (1, 64, 16, 3, 1, None, 3.0),
                                                       (700, 256, 48, 12, 4, (2, 1), 0.9), (5, 136, 20, 4, 4, (4, 4), 0.7)])
def test_routed_clamped_experts(T, H, I, E, top, groups, limit, dtype):
    """The whole feed-forward part against the plain one; in bfloat16 every expert is chosen, so no rounding changes a choice."""
    from airun_b200.parts.base import make_part
    g = torch.Generator().manual_seed(T)
    if dtype == torch.bfloat16:
        top, groups = E, (groups[0], groups[0]) if groups else None
    mlp = P.moe(I, limit, E, top, groups)
    W = {"p.router": 2 * torch.randn(E, H, generator=g) / math.sqrt(H)}
    for e in range(E):
        W.update({f"p.e{e}.{n}": 2 * torch.randn(I, H, generator=g) / math.sqrt(H) for n in ("gate", "up")})
        W[f"p.e{e}.down"] = torch.randn(H, I, generator=g) / math.sqrt(I)
    W = {n: P.to_bf16_and_back(t) for n, t in W.items()}
    gr = groups or (1, 1)
    part = make_part("feed_forward", "routed_experts", prefix="p", hidden_size=H, intermediate_size=I, num_experts=E, top=top, scores="sigmoid",
                     weight_on="output", expert="clamped_glu", limit=limit, routing="grouped", groups=gr[0], keep_groups=gr[1], group_best=2,
                     dtype=dtype, device="cuda")
    part.load_weights({s.name: dev(W[s.name], dtype) for s in part.weight_specs()})
    h = P.to_bf16_and_back(torch.randn(T, H, generator=g))
    ctx = batch_ctx([(0, T)])
    out = part.forward(ctx, dev(h, dtype))
    assert int(ctx.err.item()) == 0
    want = P.plain_moe(h.double(), {n: t.double() for n, t in W.items()}, "p", mlp, rnd=P.to_bf16_and_back if dtype == torch.bfloat16 else None)
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol), float((out.cpu().double() - want).abs().max())


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("portion", [1, 2, 37])
def test_delta_rule_half_with_columns_of_a_wider_product(portion, dtype):
    """The part's split form: handed strided columns of a product over several parts' matrices, in another slot's company,
    cut into portions; its heads times ``out_scale`` in a column slice."""
    from airun_b200.parts.base import make_part
    heads, kvh, D, Dv, taps, H, n = 4, 2, 12, 20, 3, 64, 37
    layer = P.parallel_layer((2, 1, 8, 8, 0.5, 4, 50.0), (heads, kvh, D, Dv, taps))
    W = {k: v.float() for k, v in P.random_weights(P.make_config(50, H, [layer]), seed=3).items() if ".right." in k}
    part = make_part("mixer", "gated_delta_rule", prefix="l0.mix.right", hidden_size=H, num_heads=heads, num_kv_heads=kvh, key_dim=D, value_dim=Dv,
                     conv_taps=taps, norm_eps=1e-5, decay="head", gate="silu", out_scale=0.7, dtype=dtype, device="cuda")
    part.load_weights({s.name: dev(W[s.name], torch.float32 if s.storage == "float32" else dtype) for s in part.weight_specs()})
    h = P.to_bf16_and_back(torch.randn(n, H, generator=torch.Generator().manual_seed(4)))
    state = torch.zeros(3, part.cache_spec().shape[0], device="cuda")
    got = []
    for a in range(0, n, portion):
        e = min(n, a + portion)
        ctx = batch_ctx([(a, e)], [2])
        wide = torch.zeros(e - a, part.w_in.shape[0] + 12, device="cuda")
        wide[:, 8:8 + part.w_in.shape[0]] = dev(h[a:e]) @ part.w_in.float().T
        act = torch.zeros(e - a, heads * Dv + 16, device="cuda", dtype=dtype)
        part.forward_core(ctx, None, act[:, 8:8 + heads * Dv], SimpleNamespace(state=state), proj=wide[:, 8:8 + part.w_in.shape[0]])
        assert int(ctx.err.item()) == 0 and float(act[:, :8].abs().max()) == 0
        got.append(act[:, 8:8 + heads * Dv].float().cpu().double())
    Wd = {k: v.double() for k, v in W.items()}
    Wd["l0.mix.right.o"] = 0.7 * torch.eye(heads * Dv, dtype=F64)
    want = P.plain_delta(h.double(), Wd, "l0.mix.right", layer["mixer"]["right"], 1e-5)
    tol = 5e-5 if dtype == torch.float32 else 2e-2
    assert torch.allclose(torch.cat(got), want, atol=tol, rtol=tol), float((torch.cat(got) - want).abs().max())
    assert float(state[:2].abs().max()) == 0.0


# ----------------------------------------------------------------------------- whole models
@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_whole_prompts_with_the_residual_after_every_layer(folders, name, dtype):
    folder, cfg, W, page = pick(folders, name, dtype)
    eng = engine(folder, dtype, page)
    layers = {}
    eng.model.layer_hook = lambda ci, x: layers.__setitem__(ci, x.float().cpu().numpy().copy())
    for n in (1, 2, 45, 130):
        s = random_tokens(n, cfg["vocab"], 10 + n)
        got = run_schedule(eng, [s], [[(0, n)]])[0]
        compare(got, cfg, W, s, dtype, f"{name} whole prompt of {n}")
        if dtype == "float32":
            after = []
            P.plain_forward(cfg, W, s, residuals=after)
            for ci in range(len(after)):
                assert np.allclose(layers[ci][:n], after[ci].numpy(), atol=2e-4, rtol=2e-5), (name, ci)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_prompt_then_single_tokens_and_from_the_first_token(folders, name, dtype):
    folder, cfg, W, page = pick(folders, name, dtype)
    eng = engine(folder, dtype, page)
    s = random_tokens(97, cfg["vocab"], 3)
    got = run_schedule(eng, [s], [[(0, 40)]] + [[(0, 1)]] * 57)[0]
    compare(got, cfg, W, s, dtype, f"{name} prompt then single tokens")
    s = random_tokens(30, cfg["vocab"], 4)
    got = run_schedule(eng, [s], [[(0, 1)]] * 30)[0]
    compare(got, cfg, W, s, dtype, f"{name} decoded from the first token")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_portions_of_every_size(folders, name, dtype):
    folder, cfg, W, page = pick(folders, name, dtype)
    eng = engine(folder, dtype, page)
    s = random_tokens(140, cfg["vocab"], 5)
    for cuts in ([2] * 70, [3, 5, 7, 11, 13, 17, 19, 23, 29, 13], [64, 2, 2, 1, 1, 70], [16, 17, 15, 33, 31, 8, 20]):
        assert sum(cuts) == 140
        got = run_schedule(eng, [s], [[(0, n)] for n in cuts])[0]
        compare(got, cfg, W, s, dtype, f"{name} portions {cuts[:4]}")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_unequal_requests_through_few_slots_and_pages(folders, name, dtype):
    """Six requests through three slots and a pool that holds about two of them: pages and state slots are freed and
    used again; each request's logits equal the plain ones and those of the request run alone."""
    folder, cfg, W, page = pick(folders, name, dtype)
    lens = [61, 9, 100, 33, 2, 77]
    seqs = [random_tokens(n, cfg["vocab"], 20 + n) for n in lens]
    eng = engine(folder, dtype, page, tokens=208, batch=128, reqs=3)
    schedule = [[(0, 17), (1, 9)], [(0, 30), (2, 64)], [(0, 1), (2, 2), (3, 5)], [(0, 13), (2, 34), (3, 1)], [(3, 27), (4, 2)],
                [(5, 50)], [(5, 1)], [(5, 26)]]
    got = run_schedule(eng, seqs, schedule)
    alone = engine(folder, dtype, page, tokens=208, batch=128, reqs=3)
    for i, s in enumerate(seqs):
        compare(got[i], cfg, W, s, dtype, f"{name} request {i} in the batch")
        single = run_schedule(alone, [s], [[(0, len(s))]])[0]
        if dtype == "float32":
            assert np.allclose(got[i], single, atol=3e-4, rtol=1e-4), (name, i)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    folder, cfg, W, page = pick(folders, "p2", dtype)
    eng = engine(folder, dtype, page, tokens=640)
    s = random_tokens(420, cfg["vocab"], 8)
    got = run_schedule(eng, [s], [[(0, 20)]] + [[(0, 1)]] * 400)[0]
    compare(got, cfg, W, s, dtype, "p2 four hundred single tokens")


@gpu
def test_long_contexts_beside_short_ones_in_batches_of_single_tokens(folders):
    """An engine made for long contexts cuts the keys of a single token into slices; four requests of very different
    lengths decode together, their steps replayed from graphs."""
    folder, cfg, W, page = pick(folders, "p2", "bfloat16")
    eng = engine(folder, "bfloat16", page, tokens=2048, batch=1024)
    lens = [900, 3, 270, 64]
    seqs = [random_tokens(n + 8, cfg["vocab"], 60 + n) for n in lens]
    got = run_schedule(eng, seqs, [[(i, n)] for i, n in enumerate(lens)] + [[(i, 1) for i in range(4)]] * 8)
    for i, s in enumerate(seqs):
        compare(got[i], cfg, W, s, "bfloat16", f"request {i} of {lens[i]} tokens and eight single ones")


ORDERS = {
    "one kind alone: latent": P.make_config(96, 64, [P.latent_layer(2, 16, 8, 8, 16, 0.4, mlp=P.moe(16, 1.0, 4, 2, (2, 1))), P.latent_layer(3, 8, 4, 24, 8, 0.4)]),
    "one kind alone: attention": P.make_config(96, 64, [P.attention_layer(2, 1, 16, 8, 0.4, temp=(1.0, 1)), P.attention_layer(4, 4, 8, 16, 0.4, mlp=P.moe(32, 1.0, 2, 2))]),
    "one kind alone: parallel": P.make_config(80, 48, [P.parallel_layer((2, 2, 16, 8, 0.4, 16, 20.0), (2, 2, 16, 16, 3), mlp=P.moe(32, 2.0, 4, 3, (2, 2)))]),
    "no feed-forward anywhere": P.make_config(80, 64, [
        P.parallel_layer((2, 1, 16, 16, 0.4, 2, 20.0), (1, 1, 8, 16, 2)), P.attention_layer(2, 1, 16, 16, 0.3),
        P.latent_layer(2, 8, 8, 8, 24, 0.4), P.parallel_layer((1, 1, 8, 8, 0.4, 8, 20.0), (3, 1, 8, 8, 5))]),
}


@gpu
@pytest.mark.parametrize("which", list(ORDERS))
def test_other_orders_of_layers(which, tmp_path):
    for dtype in ("float32", "bfloat16"):
        cfg = ORDERS[which] if dtype == "float32" else P.all_experts(ORDERS[which])
        W = P.random_weights(cfg, seed=len(which))
        folder = P.write_folder(str(tmp_path / dtype), cfg, W)
        s = random_tokens(70, cfg["vocab"], 9)
        eng = engine(folder, dtype, 8)
        got = run_schedule(eng, [s], [[(0, 33)], [(0, 2)], [(0, 1)], [(0, 34)]])[0]
        compare(got, cfg, W, s, dtype, which)


@gpu
def test_a_far_token_reaches_the_logits(folders):
    """A prompt of 500 tokens and the same one with ONE early token changed: the plain logits of the last rows differ by far
    more than the float32 bound, and the engine follows both, decoded and in a portion."""
    folder, cfg, W, page = folders["p2"]
    s = random_tokens(500, cfg["vocab"], 70)
    t = list(s)
    t[2] = (t[2] + 1) % cfg["vocab"]
    diff = np.abs(plain_logits(cfg, W, s)[-8:] - plain_logits(cfg, W, t)[-8:]).max()
    assert diff > 20 * 2e-4 * np.abs(plain_logits(cfg, W, s)[-8:]).max()
    for seq in (s, t):
        for cuts in ([[(0, 492)]] + [[(0, 1)]] * 8, [[(0, 250)], [(0, 250)]]):
            eng = engine(folder, "float32", page, tokens=512, batch=512)
            compare(run_schedule(eng, [seq], cuts)[0], cfg, W, seq, "float32", "far token")


@gpu
def test_greedy_generation_through_the_engine(folders):
    """Through the engine's own entry points and scheduler: add_request / run_step for unequal requests at once, and
    generate."""
    import airun_b200
    folder, cfg, W, page = folders["p1"]
    eng = engine(folder, "float32", page)
    prompts = [random_tokens(n, cfg["vocab"], 40 + n) for n in (5, 23, 1)]
    reqs = [eng.add_request(p, airun_b200.SamplingParams.greedy(), max_new_tokens=12) for p in prompts]
    while eng.scheduler.has_work():
        eng.run_step()
    for p, r in zip(prompts, reqs):
        assert r.output == P.plain_greedy(cfg, W, p, 12)
    one = eng.generate(prompts[1], airun_b200.SamplingParams.greedy(), max_new_tokens=12)
    assert one.token_ids == P.plain_greedy(cfg, W, prompts[1], 12)
    eng.manager.check_invariants()


@gpu
def test_replay_tool_on_a_folder(folders, tmp_path):
    folder, cfg, W, page = folders["p2"]
    a, b = random_tokens(50, cfg["vocab"], 1), random_tokens(21, cfg["vocab"], 2)
    r = Replay(folder, "float32", str(tmp_path / "out"), max_tokens=128)
    try:
        r1 = r.step([{"id": "a", "tokens": a[:30], "want": [0, 29]}])
        r2 = r.step([{"id": "a", "tokens": a[30:49], "want": []}, {"id": "b", "tokens": b, "want": [20]}], end=["b"])
        r3 = r.step([{"id": "a", "tokens": a[49:], "want": [0]}], end=["a"])
    finally:
        r.close()
    la, lb = P.plain_forward(cfg, W, a).numpy(), P.plain_forward(cfg, W, b).numpy()
    assert_close(np.concatenate([r1, r2, r3]), np.stack([la[0], la[29], lb[20], la[49]]).astype(np.float32), "float32", "replay")
