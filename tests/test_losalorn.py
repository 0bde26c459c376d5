"""The Losalorn decoder in the engine against the plain implementation (tests/plain_losalorn.py): each mechanism's
kernels alone, then whole models of several small shapes through the step function, the scheduler and the replay tool:
whole prompts, token-by-token decoding, portions down to two tokens, unequal batches, slots and pages used again, far
keys, page borders, window edges, the first tokens, long decoding, loops of other lengths and other orders of layers."""
from __future__ import annotations

import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_losalorn as P
from helpers import Replay, assert_close, bf16_noise, random_tokens

F64 = torch.float64
gpu = pytest.mark.gpu


# ----------------------------------------------------------------------------- small shapes
def shape_l1() -> dict:
    """Odd sizes everywhere (a width no tensor-core product takes): groups of three query heads, q/k heads shared by two
    state heads, a window of 11 over pages of 8, a rotation whose scaled frequencies fall on both sides of the bands, an
    attention without window or scaling that rotates its whole head, a convolution of one tap, layers with and without
    a feed-forward, a loop in the middle that runs three times."""
    return P.make_config(vocab=150, width=100, eps=3e-5, emb_scale=2.5, cap=9.0, loop=(1, 3, 3), layers=[
        P.delta_layer(4, 2, 12, 20, conv=3, mlp=P.dense(72, 0.8)),
        P.attention_layer(3, 1, 10, window=11, rot=6, base=300.0, scaling=(4.0, 1.0, 4.0, 64), scale=0.4),
        P.delta_layer(2, 2, 40, 7, conv=1),
        P.attention_layer(2, 2, 12, rot=12, base=1000.0, mlp=P.dense(40, 1.5))])


def shape_l2() -> dict:
    """Sizes the tensor-core kernels take in bfloat16: heads of 64 and 32, groups of four and of one, a window of 40 over
    pages of 16, a loop from the first layer on, twice."""
    return P.make_config(vocab=192, width=128, emb_scale=4.0, cap=20.0, loop=(0, 2, 2), layers=[
        P.attention_layer(4, 1, 64, window=40, rot=16, base=10000.0, scaling=(8.0, 1.0, 4.0, 256), scale=0.2, mlp=P.dense(160, 1.0)),
        P.delta_layer(4, 1, 16, 32, conv=4),
        P.attention_layer(4, 4, 32, window=17, rot=32, base=500.0, mlp=P.dense(96, 2.0)),
        P.delta_layer(2, 1, 64, 48, conv=2, mlp=P.dense(64, 0.7))])


def shape_l3() -> dict:
    """Without a loop, a rotation or a cap; a delta rule first and last; one head, taps above the page size."""
    cfg = P.make_config(vocab=64, width=48, emb_scale=1.0, layers=[
        P.delta_layer(1, 1, 8, 8, conv=9),
        P.attention_layer(2, 1, 8, window=200, mlp=P.dense(32, 1.0)),
        P.delta_layer(3, 3, 16, 8, conv=2)])
    del cfg["logit_softcap"]
    return cfg


def shape_l4() -> dict:
    """A loop over all layers that runs once (the stream is mixed all the same), head sizes of 40 and 72 that need
    padding, rotated parts of 4 and 8 dimensions, a window of one token."""
    return P.make_config(vocab=130, width=96, emb_scale=7.0, cap=15.0, loop=(0, 3, 1), layers=[
        P.attention_layer(4, 2, 72, window=33, rot=8, base=50.0, scaling=(2.0, 0.5, 8.0, 40), mlp=P.dense(48, 1.0)),
        P.attention_layer(2, 2, 40, window=1, rot=4, base=70.0),
        P.delta_layer(6, 2, 24, 16, conv=3, mlp=P.dense(80, 1.2))])


SHAPES = {"l1": (shape_l1, 8), "l2": (shape_l2, 16), "l3": (shape_l3, 8), "l4": (shape_l4, 16)}      # configuration, page size


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, (make, page) in SHAPES.items():
        cfg = make()
        W = P.random_weights(cfg, seed=len(name) * 11 + ord(name[-1]))
        out[name] = (P.write_folder(str(tmp_path_factory.mktemp(name)), cfg, W), cfg, W, page)
    return out


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


def plain_logits(cfg, W, seq, rnd=None):
    """The plain logits of a sequence, kept for the next test that asks for the same ones."""
    key = (json.dumps(cfg, sort_keys=True), id(W), tuple(seq), rnd is None)
    if key not in _PLAIN:
        _PLAIN[key] = (P.plain_forward(cfg, W, seq, rnd=rnd).numpy(), W)         # W is held, so that its id stays its own
    return _PLAIN[key][0]


def compare(got, cfg, W, seq, dtype, what):
    exact = plain_logits(cfg, W, seq)
    if dtype == "float32":
        return assert_close(got, exact.astype(np.float32), dtype, what)
    rounded = plain_logits(cfg, W, seq, P.to_bf16_and_back)
    # the engine's rounding is another draw of the same noise, amplified by every pass of a loop: a row is held to three
    # times its own noise, where helpers.assert_close alone would hold it to two
    assert_close(got, rounded.astype(np.float32), dtype, what, 1.5 * bf16_noise(rounded, exact))


# ----------------------------------------------------------------------------- without a GPU
def test_config_reads_sizes_constants_and_the_loop():
    from airun_b200.config import LosalornConfig, architecture_name, lookup_architecture
    d = shape_l1()
    assert architecture_name(d) == "Losalorn" and lookup_architecture("Losalorn")[0] is LosalornConfig
    c = LosalornConfig.from_dict(d)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embedding_scale, c.logit_softcap) == (150, 100, 3e-5, 2.5, 9.0)
    assert [(o.layer, o.reinject, o.cache_from) for o in c.execution_order()] == [
        (0, False, None), (1, True, None), (2, False, None), (1, True, None), (2, False, None), (1, True, None), (2, False, None),
        (3, False, None)]
    assert c.residual_input() == ("mix_with_embedding", "loop.in", dict(hidden_size=100)) and c.tie_word_embeddings
    assert c.embedding() == ("token_embedding", dict(scale=2.5)) and c.head() == ("lm_head", dict(soft_cap=9.0))
    specs = c.layer_specs()
    assert [s.mixer for s in specs] == ["gated_delta_rule", "softmax_attention", "gated_delta_rule", "softmax_attention"]
    assert [s.feed_forward for s in specs] == ["clamped_glu", "", "", "clamped_glu"] and all(s.arrangement == "sandwich" for s in specs)
    a = specs[0].mixer_args
    assert (a["num_heads"], a["num_kv_heads"], a["key_dim"], a["value_dim"], a["conv_taps"], a["decay"], a["gate"]) == (4, 2, 12, 20, 3, "head", "silu")
    b = specs[1].mixer_args
    assert (b["window"], b["scale"], b["values"], b["sink"], b["position"]) == (11, 0.4, "keys", "one", "rotary_neox_by_wavelength")
    assert b["position_args"] == dict(rotary_dim=6, theta=300.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=64.0))
    assert specs[3].mixer_args["window"] == 0 and specs[3].mixer_args["position_args"]["scaling"] is None
    assert specs[3].mixer_args["scale"] == pytest.approx(12 ** -0.5) and specs[0].ffn_args["limit"] == 0.8
    assert c.ignorable_tensors() == ["l1.norm2", "l1.norm2b", "l2.norm2", "l2.norm2b"]
    assert LosalornConfig.from_dict(c.to_dict()) == c
    p = LosalornConfig.from_dict(shape_l3())
    assert p.residual_input() is None and p.logit_softcap is None and "loop.in" in p.ignorable_tensors()
    assert not any(o.reinject for o in p.execution_order()) and p.layer_specs()[1].mixer_args["position"] == "none"
    once = LosalornConfig.from_dict(shape_l4())
    assert [(o.layer, o.reinject) for o in once.execution_order()] == [(0, True), (1, False), (2, False)]
    assert LosalornConfig.from_dict(dict(shape_l4(), loop=dict(start=0, stop=3, times=0))).execution_order() == []


def test_config_lists_every_problem():
    from airun_b200.config import ConfigError, LosalornConfig
    d = shape_l1()
    d["layers"][0]["mixer"]["kv_heads"] = 3
    d["layers"][0]["mlp"]["limit"] = 0
    d["layers"][1]["mixer"]["vdim"] = 12
    d["layers"][1]["mixer"]["rot"]["scaling"]["high"] = 0.5
    d["layers"][2]["type"] = "other"
    d["layers"][3]["mixer"]["rot"]["dims"] = 14
    d["loop"]["stop"] = 9
    d["norm"]["eps"] = 0
    with pytest.raises(ConfigError) as e:
        LosalornConfig.from_dict(d)
    for piece in ("layers[0].mixer.heads", "layers[0].mlp.limit", "layers[1].mixer.vdim (12) must equal dim", "scaling.high must be at least low",
                  "layers[2] needs", "layers[3].mixer.rot.dims", "loop must satisfy", "norm.eps"):
        assert piece in str(e.value), piece


def test_declared_tensors_are_the_files_tensors():
    from airun_b200.config import LosalornConfig
    from airun_b200.engine.model import DecoderModel
    for name, (make, _) in SHAPES.items():
        m = DecoderModel(LosalornConfig.from_dict(make()), torch.float32, "cpu")
        declared = {s.name: tuple(s.shape) for s in m.weight_specs()}
        shapes = P.tensor_shapes(make())
        assert declared == shapes, (name, set(declared) ^ set(shapes))


def test_every_pass_owns_its_cache_and_a_row_is_key_and_value():
    from airun_b200.cache.manager import CacheManager
    from airun_b200.config import LosalornConfig
    from airun_b200.engine.model import DecoderModel
    from airun_b200.parts.base import PagedKVSpec, StateSpec
    m = DecoderModel(LosalornConfig.from_dict(shape_l1()), torch.float32, "cpu")
    specs, src = m.cache_specs()
    assert src == [None] * 8
    small, state2 = PagedKVSpec(1, 16, 11, values=False), StateSpec((2 * 40 * 7,), torch.float32)      # key of 10 and 6 unrotated dimensions; no tail for one tap
    assert specs == [StateSpec((4 * 12 * 20 + 2 * (2 * 24 + 80),), torch.float32), small, state2, small, state2, small, state2,
                     PagedKVSpec(2, 24, 0, values=False)]
    mgr = CacheManager(specs, src, page_size=8, num_pages=12, max_requests=3)
    b = mgr.bindings
    assert [x.kind for x in b] == ["state", "paged", "state", "paged", "state", "paged", "state", "paged"]
    assert b[1].gid == b[3].gid == b[5].gid != b[7].gid and [b[i].index for i in (1, 3, 5)] == [0, 1, 2]
    assert b[2].gid == b[4].gid == b[6].gid and [b[i].index for i in (2, 4, 6)] == [0, 1, 2]
    mgr.add_request("a")
    mgr.reserve("a", 40)
    mgr.commit("a", 40)
    free = mgr.free_pages()
    assert free[b[7].gid] == 7 and free[b[1].gid] == 10           # the window's pages go back as it passes
    mgr.free_request("a")
    assert set(mgr.free_pages().values()) == {12}


def test_frequencies_of_the_position_part():
    """Against the plain formula, with wavelengths on both sides of both bands, on a band's edge, and equal bands."""
    from airun_b200.parts.base import make_part
    for dims, base, sc in ((20, 30000.0, (6.0, 1.0, 3.0, 2048)), (64, 500.0, (8.0, 0.5, 8.0, 100)), (8, 10.0, (3.0, 2.0, 2.0, 50)),
                           (2, 7.0, (3.0, 1.0, 4.0, 2 * math.pi)), (12, 1000.0, None), (32, 10.0, (5.0, 1.0, 2.0, 1e6)), (32, 10.0, (5.0, 1.0, 2.0, 2))):
        scaling = None if sc is None else dict(factor=sc[0], low=sc[1], high=sc[2], original=sc[3])
        part = make_part("position", "rotary_neox_by_wavelength", rotary_dim=dims, theta=base, scaling=scaling)
        want = torch.tensor(P.plain_frequencies(dims, base, scaling), dtype=F64)
        kind, rdim, inv = part.fused()
        from airun_b200.kernels import ops
        assert kind == ops.ROPE_NEOX and rdim == dims and torch.allclose(inv.double(), want, rtol=1e-6)
    bands = P.plain_frequencies(20, 30000.0, dict(factor=6.0, low=1.0, high=3.0, original=2048))
    plain = P.plain_frequencies(20, 30000.0, None)
    ratio = [a / b for a, b in zip(bands, plain)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 6) and any(0.17 < r < 1.0 for r in ratio)


def test_plain_mechanisms_against_hand_worked_cases():
    # the softmax with a one in its denominator: one score of ln 3 weighs 3/4, two scores of 0 weigh 1/3 each
    p = P.plain_softmax_plus_one(torch.tensor([[math.log(3.0), -math.inf], [0.0, 0.0]], dtype=F64))
    assert torch.allclose(p, torch.tensor([[0.75, 0.0], [1 / 3, 1 / 3]], dtype=F64))
    assert torch.allclose(P.plain_softmax_plus_one(torch.tensor([[-800.0, -900.0], [900.0, 0.0]], dtype=F64)), torch.tensor([[0.0, 0.0], [1.0, 0.0]], dtype=F64))
    # the rotation pairs i with i + dims/2 and leaves the rest
    x = torch.randn(5, 2, 6, dtype=F64)
    r = P.plain_rotate_half(x, torch.arange(5), 4, [1.0, 0.1])
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])
    assert float(r[3, 0, 1]) == pytest.approx(float(x[3, 0, 1] * math.cos(0.3) - x[3, 0, 3] * math.sin(0.3)))
    assert float(r[3, 0, 3]) == pytest.approx(float(x[3, 0, 3] * math.cos(0.3) + x[3, 0, 1] * math.sin(0.3)))
    # the window: the query itself and size - 1 before it
    w = P.plain_window(6, 3)
    assert w.sum(-1).tolist() == [1, 2, 3, 3, 3, 3] and w[5].tolist() == [False] * 3 + [True] * 3
    # the gated unit: the gate has no lower clamp
    g, u = torch.tensor([5.0, -30.0, 0.5], dtype=F64), torch.tensor([9.0, -9.0, 0.25], dtype=F64)
    want = [2 / (1 + math.exp(-3.404)) * 3, -30 / (1 + math.exp(1.702 * 30)) * -1, 0.5 / (1 + math.exp(-0.851)) * 1.25]
    assert torch.allclose(P.plain_clamped_unit(g, u, 2.0), torch.tensor(want, dtype=F64))
    # the pass input reads the stream first
    assert P.plain_pass_input(torch.tensor([[1.0, 2.0]]), torch.tensor([[10.0, 20.0]]), torch.tensor([[1.0, 0, 0, 1], [0, 1, 1, 0]])).tolist() == [[21.0, 12.0]]
    # the recurrence: carried across a cut; a unit key with beta 1 replaces what it predicts; the read-out sees the write
    gen = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(12, 2, n, generator=gen, dtype=F64) for n in (3, 3, 4))
    dec, beta = torch.rand(12, 2, generator=gen, dtype=F64), torch.rand(12, 2, generator=gen, dtype=F64)
    o, S = P.plain_delta_recurrence(q, k, v, dec, beta)
    o1, S1 = P.plain_delta_recurrence(q[:5], k[:5], v[:5], dec[:5], beta[:5])
    o2, S2 = P.plain_delta_recurrence(q[5:], k[5:], v[5:], dec[5:], beta[5:], state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
    kk = torch.zeros(12, 2, 3, dtype=F64)
    kk[..., 1] = 1.0
    o3, _ = P.plain_delta_recurrence(kk, kk, v, dec, torch.ones(12, 2, dtype=F64))
    assert torch.allclose(o3, v)
    assert P.plain_head_decay(torch.tensor([[0.0]]), torch.tensor([0.0]), torch.tensor([0.0])).item() == pytest.approx(0.5)
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


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,n", [(5, 100), (1, 48), (90, 328), (3, 2051), (70, 2048), (2, 4096), (66, 9001), (3, 20000)])
def test_norms_on_both_sides_in_one_pass(T, n, dtype):
    from airun_b200.kernels import ops
    g = torch.Generator().manual_seed(T + n)
    x, y = 3 * torch.randn(T, n, generator=g), torch.randn(T, n, generator=g) * torch.rand(T, 1, generator=g)
    a, b = 1 + 0.3 * torch.randn(n, generator=g), 1 + 0.3 * torch.randn(n, generator=g)
    v = x.double() + P.plain_rmsnorm(y.double(), a.double(), 1e-4)
    h = P.plain_rmsnorm(v, b.double(), 1e-3)
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    xd, out = dev(x), torch.empty(T, n, device="cuda", dtype=dtype)
    ops.sandwich_norm(xd, out, y=dev(y), w_post=dev(a), eps_post=1e-4, w_pre=dev(b), eps_pre=1e-3)
    assert torch.allclose(xd.cpu().double(), v, rtol=2e-6, atol=2e-6)
    assert torch.allclose(out.cpu().double(), h, rtol=tol * 4, atol=tol * 4)
    # chosen rows: x stays as it is
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device="cuda")
    xd, few = dev(x), torch.empty(3, n, device="cuda", dtype=dtype)
    ops.sandwich_norm(xd, few, y=dev(y), w_post=dev(a), eps_post=1e-4, w_pre=dev(b), eps_pre=1e-3, rows=rows)
    assert torch.equal(xd.cpu(), x)
    assert torch.allclose(few.cpu().double(), h[rows.long().cpu()], rtol=tol * 4, atol=tol * 4)
    # the norm and the add alone; the copy and the split, with and without something to add
    ops.sandwich_norm(xd, None, y=dev(y), w_post=dev(a), eps_post=1e-4)
    assert torch.allclose(xd.cpu().double(), v, rtol=2e-6, atol=2e-6)
    xd = dev(x)
    if dtype == torch.float32:
        ops.sandwich_norm(xd, out, mode=ops.SANDWICH_COPY, write_back=False)
        assert torch.equal(out.cpu(), x)
        ops.sandwich_norm(xd, out, y=dev(y), w_post=dev(a), eps_post=1e-4, mode=ops.SANDWICH_COPY, write_back=False)
        assert torch.allclose(out.cpu().double(), v, rtol=2e-6, atol=2e-6) and torch.equal(xd.cpu(), x)
    else:
        two = torch.empty(T, 2 * n, device="cuda", dtype=dtype)
        ops.sandwich_norm(xd, two, y=dev(y), w_post=dev(a), eps_post=1e-4, mode=ops.SANDWICH_SPLIT, write_back=False)
        hi, lo = two[:, :n].double().cpu(), two[:, n:].double().cpu()
        assert torch.allclose(hi + lo, v, rtol=2.0 ** -15, atol=1e-6) and torch.equal(xd.cpu(), x)
        assert float(lo.abs().max()) > 0 and torch.allclose(hi, v, rtol=2.0 ** -8, atol=1e-5)
    # a row without content stays finite
    z = torch.zeros(1, n, device="cuda")
    ops.sandwich_norm(z, out[:1], y=torch.zeros(1, n, device="cuda"), w_post=dev(a), eps_post=1e-4, w_pre=dev(b), eps_pre=1e-3)
    assert float(out[0].abs().max()) == 0.0


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H", [(5, 100), (300, 128), (17, 96)])
def test_stream_mixed_with_the_embedding(T, H, dtype):
    """x <- Mx x + M0 x0 with what the block before left pending carried out first; also on the bfloat16 path the stream is
    not rounded to bfloat16 on its way through the product."""
    from airun_b200.parts.base import PostNormWrite, make_part
    g = torch.Generator().manual_seed(H)
    part = make_part("residual_input", "mix_with_embedding", prefix="loop.in", hidden_size=H, dtype=dtype, device="cuda")
    w = P.to_bf16_and_back(torch.randn(H, 2 * H, generator=g) / math.sqrt(2 * H))
    part.load_weights({"loop.in": dev(w, dtype)})
    x0, x, y = (4 * torch.randn(T, H, generator=g) for _ in range(3))
    a = 1 + 0.3 * torch.randn(H, generator=g)
    ctx = batch_ctx([(0, T)])
    kept = part.begin(ctx, dev(x0))
    want = P.plain_pass_input(x.double() + P.plain_rmsnorm(y.double(), a.double(), 1e-4), x0.double(), w.double())
    bound = 2e-5 if dtype == torch.float32 else 4e-4                  # bfloat16 rounding of x alone would be off by 2e-2
    for pending, target in ((PostNormWrite(dev(y), dev(a), 1e-4), want),
                            (None, P.plain_pass_input(x.double(), x0.double(), w.double())),
                            (dev(y), P.plain_pass_input((x + y).double(), x0.double(), w.double()))):
        xd = dev(x)
        rest = part.forward(ctx, xd, pending, kept)
        assert torch.allclose((xd + rest).cpu().double(), target, atol=bound, rtol=bound), float(((xd + rest).cpu().double() - target).abs().max())


def attention_case(seq_lens, new_lens, nh, nkv, D, page, dtype, seed, rot=None, bias=False, spike=None):
    """Rows written through the prologue kernel (pages handed out in a scrambled order) for the first len - new tokens of
    every request, then the last ``new`` tokens of each as one batch.  ``rot``: (dims, base, scaling) or None.  Returns the
    projections, the biases, the cache and the last batch's (spans, ctx, q, live requests)."""
    from airun_b200.kernels import ops
    from airun_b200.parts.base import make_part
    g = torch.Generator().manual_seed(seed)
    width = (nh + nkv) * D
    reqs = []
    for n in seq_lens:
        proj = torch.randn(n, width, generator=g)
        if spike is not None:
            spike(proj, n)
        reqs.append(proj)
    b = 0.5 * torch.randn(width, generator=g) if bias else None
    kind, r, inv = ops.ROPE_NONE, 0, None
    if rot:
        kind, r, inv = make_part("position", "rotary_neox_by_wavelength", rotary_dim=rot[0], theta=rot[1], scaling=rot[2], device="cuda").fused()
    blocks = [(n + page - 1) // page for n in seq_lens]
    num_pages = sum(blocks) + 3
    perm = torch.randperm(num_pages, generator=g).tolist()
    bt = torch.full((len(seq_lens), max(blocks)), -1, dtype=torch.int32)
    for i, nb in enumerate(blocks):
        for blk in range(nb):
            bt[i, blk] = perm.pop()
    cache = SimpleNamespace(pool=torch.zeros(num_pages, nkv * page * (D + r), device="cuda", dtype=dtype), block_table=bt.cuda(),
                            page_size=page, shared=False)
    last = None
    for phase in (0, 1):
        spans = [(0, n - m) if phase == 0 else (n - m, n) for n, m in zip(seq_lens, new_lens)]
        live = [(i, s) for i, s in enumerate(spans) if s[1] > s[0]]
        if not live:
            continue
        ctx = batch_ctx([s for _, s in live])
        table = cache.block_table
        cache.block_table = table[[i for i, _ in live]].contiguous()
        proj = dev(torch.cat([reqs[i][a:e] for i, (a, e) in live]))
        q = torch.empty(proj.shape[0], nh * D, device="cuda", dtype=dtype)
        ops.qkv_prepare(proj, None if b is None else dev(b), None, None, False, 1e-5, kind, r, inv, 0.0, 0, q, cache, ctx, nh, nkv, D, D,
                        store=True, one_row=True)
        assert int(ctx.err.item()) == 0
        last = ([s for _, s in live], ctx, q, [i for i, _ in live])
        if phase == 0:
            cache.block_table = table
    return reqs, b, cache, last


def plain_qkv(proj, b, nh, nkv, D, rot):
    n = proj.shape[0]
    p = proj.double() + (b.double() if b is not None else 0.0)
    q, k = p[:, :nh * D].view(n, nh, D), p[:, nh * D:].view(n, nkv, D)
    v = k
    if rot:
        f = P.plain_frequencies(rot[0], rot[1], rot[2])
        q, k = P.plain_rotate_half(q, torch.arange(n), rot[0], f), P.plain_rotate_half(k, torch.arange(n), rot[0], f)
    return q, k, v


def plain_case(reqs, b, spans, live, nh, nkv, D, scale, rot, window, sink=True):
    """[rows of the last batch, heads, D] in the order of the values' own dimensions."""
    outs = []
    for i, (a, e) in zip(live, spans):
        q, k, v = plain_qkv(reqs[i][:e], b, nh, nkv, D, rot)
        vis = P.plain_window(e, window)
        o = torch.zeros(e, nh, D, dtype=F64)
        for h in range(nh):
            kv = h // (nh // nkv)
            s = (q[:, h] @ k[:, kv].T * scale).masked_fill(~vis, -math.inf)
            w = P.plain_softmax_plus_one(s) if sink else torch.softmax(s, dim=-1)
            o[:, h] = w @ v[:, kv]
        outs.append(o[a:e])
    return torch.cat(outs)


def run_attention(q, cache, ctx, nh, nkv, D, scale, tail, window, sink=True, tensor_cores=False):
    """The heads' results, brought back from the cached order (dimensions tail .. D-1, 0 .. tail-1) to their own."""
    from airun_b200.kernels import fast, ops
    zero = torch.zeros(nh, device="cuda") if sink else None
    wide = torch.zeros(q.shape[0], nh * D + 16, device="cuda", dtype=q.dtype)
    out = wide[:, 8:8 + nh * D]
    if tensor_cores:
        part = SimpleNamespace(D=D, Dv=D, nh=nh, nkv=nkv, scale=scale, table=None, sink=zero, window=window, out_scale=1.0, tail=tail)
        assert fast.softmax_attention_bf16(ctx, q, out, cache, part)
    else:
        ops.softmax_attention(q, out, cache, ctx, nh, nkv, D, D, scale, None, zero, window, 1.0, tail=tail)
    assert int(ctx.err.item()) == 0 and float(wide[:, :8].abs().max()) == 0 and float(wide[:, 8 + nh * D:].abs().max()) == 0
    o = out.float().cpu().double().view(q.shape[0], nh, D)
    return torch.cat([o[..., D - tail:], o[..., :D - tail]], dim=-1) if tail else o


SC = dict(factor=4.0, low=1.0, high=4.0, original=64)
ATT_SHAPES = [  # heads, kv heads, D, rotation, page
    (3, 1, 12, (6, 300.0, SC), 8), (4, 2, 88, (16, 500.0, None), 16), (8, 8, 32, (32, 500.0, SC), 16), (2, 1, 132, (132, 90.0, SC), 8),
    (6, 3, 64, (24, 500.0, SC), 32), (1, 1, 40, (4, 70.0, None), 16), (16, 1, 16, None, 8), (4, 1, 128, (64, 10000.0, SC), 16),
    (2, 2, 256, (256, 500.0, None), 8), (5, 1, 72, (10, 40.0, SC), 8), (4, 2, 24, (24, 40.0, None), 24)]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", ATT_SHAPES)
@pytest.mark.parametrize("bias", [False, True])
def test_cached_rows_and_attention_over_scrambled_pages(shape, bias, dtype):
    """A portion beside a whole prompt beside a single token; and the cached row itself: the rotated key, then the
    rotated dimensions as they were projected."""
    nh, nkv, D, rot, page = shape
    tail = rot[0] if rot else 0
    seqs, new, window = [70, 23, 91], [13, 23, 1], 19
    reqs, b, cache, (spans, ctx, q, live) = attention_case(seqs, new, nh, nkv, D, page, dtype, 5, rot, bias)
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    for i in live:
        qp, kp, vp = plain_qkv(reqs[i], b, nh, nkv, D, rot)
        for pos in (0, 7, 8, seqs[i] - 1):
            page_rows = cache.pool[int(cache.block_table[i, pos // page])].view(nkv, page, D + tail)[:, pos % page].double().cpu()
            assert torch.allclose(page_rows[:, :D], kp[pos], atol=tol, rtol=tol) and torch.allclose(page_rows[:, D:], vp[pos, :, :tail], atol=tol, rtol=tol)
        a, e = spans[live.index(i)]
        rows = q[int(ctx.cu_tokens[live.index(i)]):int(ctx.cu_tokens[live.index(i) + 1])].double().cpu().view(e - a, nh, D)
        assert torch.allclose(rows, qp[a:e], atol=tol, rtol=tol)
    scale = 1.5 * D ** -0.5
    for sink in (True, False):
        got = run_attention(q, cache, ctx, nh, nkv, D, scale, tail, window, sink)
        want = plain_case(reqs, b, spans, live, nh, nkv, D, scale, rot, window, sink)
        assert torch.allclose(got, want, atol=tol, rtol=tol), float((got - want).abs().max())


@gpu
@pytest.mark.parametrize("shape", [s for s in ATT_SHAPES if s[2] <= 128])
@pytest.mark.parametrize("new", [[13, 23, 1], [1, 1, 1], [130, 70, 64]])
def test_tensor_core_attention_against_the_plain_kernel_and_the_formula(shape, new):
    """A portion beside a whole prompt beside a single token; single tokens alone (700, 23 and 1500 keys, cut into
    slices, some of them empty); several tiles of several requests."""
    nh, nkv, D, rot, page = shape
    tail = rot[0] if rot else 0
    seqs = [70, 23, 91] if new == [13, 23, 1] else [700, 23, 1500] if new[0] == 1 else [300, 70, 65]
    window = 0 if new[0] == 1 else 90
    reqs, b, cache, (spans, ctx, q, live) = attention_case(seqs, new, nh, nkv, D, page, torch.bfloat16, 6, rot)
    scale = 1.5 * D ** -0.5
    want = plain_case(reqs, b, spans, live, nh, nkv, D, scale, rot, window)
    got = run_attention(q, cache, ctx, nh, nkv, D, scale, tail, window, tensor_cores=True)
    plain = run_attention(q, cache, ctx, nh, nkv, D, scale, tail, window)
    assert torch.allclose(got, want, atol=1e-1, rtol=3e-2), float((got - want).abs().max())        # bfloat16 q and rows against float64
    assert torch.allclose(got, plain, atol=2e-2, rtol=2e-2), float((got - plain).abs().max())      # the same inputs: only the weights' rounding


@gpu
@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("window", [1, 7, 8, 63, 64, 65, 100, 200])
@pytest.mark.parametrize("new", [1, 70])
def test_window_edges_key_by_key(window, new, tensor_cores):
    """The key just inside the window weighs, the key just outside does not: the scores are all zero (the queries are), and
    every one of the last keys is one hot in a dimension of its own, so the output spells out which keys a query saw."""
    n, D, page = 300, 128, 8

    def spike(proj, n_):
        proj[:, :D] = 0.0
        proj[:, D:] = torch.eye(n_, n_)[:, -D:]
    reqs, b, cache, (spans, ctx, q, live) = attention_case([n], [new], 1, 1, D, page, torch.bfloat16 if tensor_cores else torch.float32, 1, None, spike=spike)
    got = run_attention(q, cache, ctx, 1, 1, D, 1.0, 0, window, tensor_cores=tensor_cores)
    for row, i in enumerate(range(n - new, n)):
        lo = max(0, i - window + 1)
        want = torch.zeros(n, dtype=F64)
        want[lo:i + 1] = 1.0 / (i + 2 - lo)                      # one more term in the denominator
        assert torch.allclose(got[row, 0], want[-D:], atol=4e-3 if tensor_cores else 1e-6), (i, window)


@gpu
@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("key_at", [0, 7, 8, 299, 444, 599])
@pytest.mark.parametrize("new", [1, 40])
def test_one_key_that_stands_out(key_at, new, tensor_cores):
    """Among 600 keys ONE has a large score with the last query; its value (its own unrotated key) must be what the query
    returns: far back, at position 0, at a page border, and the token itself; rotated dimensions are in play."""
    n, nh, nkv, D, page, rot = 600, 2, 1, 32, 8, (8, 100.0, None)

    def spike(proj, n_):
        proj *= 0.05
        proj[n_ - 1, 20:nh * D:D] = 6.0                     # the last token's query heads point along dimension 20
        proj[key_at, nh * D + 20] = 6.0                     # and so does the key at key_at
        proj[key_at, nh * D + 3] = 2.5                      # a rotated dimension of its value
    reqs, b, cache, (spans, ctx, q, live) = attention_case([n], [new], nh, nkv, D, page, torch.bfloat16 if tensor_cores else torch.float32, 3, rot, spike=spike)
    got = run_attention(q, cache, ctx, nh, nkv, D, 1.0, rot[0], 0, tensor_cores=tensor_cores)
    v = reqs[0][key_at, nh * D:].double()
    for h in range(nh):
        assert torch.allclose(got[-1, h], v, atol=3e-2 if tensor_cores else 1e-3), (h, float((got[-1, h] - v).abs().max()))
    want = plain_case(reqs, b, spans, live, nh, nkv, D, 1.0, rot, 0)
    assert torch.allclose(got, want, atol=6e-2 if tensor_cores else 2e-5, rtol=3e-2 if tensor_cores else 1e-5)


DELTA_SHAPES = [(4, 2, 12, 20, 3), (2, 2, 130, 33, 4), (1, 1, 8, 8, 1), (4, 1, 64, 96, 2), (3, 3, 32, 64, 6), (2, 1, 128, 128, 4), (1, 1, 256, 40, 4),
                (2, 1, 64, 64, 4), (3, 1, 20, 16, 5)]


@gpu
@pytest.mark.parametrize("heads,kvh,D,Dv,taps", DELTA_SHAPES)
@pytest.mark.parametrize("long", [False, True])
def test_delta_rule_with_a_decay_per_head(heads, kvh, D, Dv, taps, long):
    """Three requests of unequal length in one batch, each cut into steps at other places (also portions shorter than the
    convolution), slots out of order, decays from 1e-20 to a hair below one; the convolution's tail and the matrices
    against the plain implementation."""
    from airun_b200.kernels import ops
    g = torch.Generator().manual_seed(heads * 100 + D)
    lens, cuts, slots = ([150, 1, 231], [[40, 41, 90], [0, 0, 0], [200, 210, 213]], [1, 0, 3]) if long else \
        ([13, 1, 37], [[2, 3, 5], [0, 0, 0], [1, 35, 36]], [2, 0, 3])
    kd, vd = kvh * D, heads * Dv
    C = 2 * kd + vd
    data = [dict(x=torch.randn(n, C, generator=g), beta=2 * torch.randn(n, heads, generator=g), a=3 * torch.randn(n, heads, generator=g) - 4.0)
            for n in lens]
    for d in data:
        d["a"][::7] = 40.0                                   # now and then a token that wipes the state
    a_log, dtb = torch.randn(heads, generator=g) * 0.5, torch.randn(heads, generator=g)
    wconv = torch.randn(C, taps, generator=g) * 0.6
    state = torch.zeros(4, heads * D * Dv + (taps - 1) * C, device="cuda")
    got = [[] for _ in lens]
    for part in range(4):
        spans = [((c[part - 1] if part else 0), (c[part] if part < 3 else n)) for n, c in zip(lens, cuts)]
        rows = [i for i, (s, e) in enumerate(spans) if e > s]
        ctx = batch_ctx([spans[i] for i in rows], [slots[i] for i in rows])
        cat = lambda key: torch.cat([data[i][key][spans[i][0]:spans[i][1]] for i in rows])
        proj = dev(torch.cat([cat("x"), cat("beta"), cat("a")], dim=1))
        T = proj.shape[0]
        conv = torch.empty(T, C, device="cuda")
        ops.short_conv(proj[:, :C], dev(wconv), state, heads * D * Dv, ctx, conv, 2 * kvh, kvh, D, 1e-6, D ** -0.5)
        o = torch.empty(T, vd, device="cuda")
        ops.recurrent_state(ops.RECURRENCE_DELTA_HEAD, conv[:, :kd], conv[:, kd:2 * kd], conv[:, 2 * kd:], proj[:, C + heads:], state, ctx, o,
                            heads, heads // kvh, D, Dv, beta=proj[:, C:C + heads], tail_src=proj[:, :C], tail_off=heads * D * Dv,
                            tail_rows=taps - 1, a_log=dev(a_log), dt_bias=dev(dtb))
        assert int(ctx.err.item()) == 0
        for j, i in enumerate(rows):
            got[i].append(o[ctx.cu_tokens[j]:ctx.cu_tokens[j + 1]].cpu())
    rep = heads // kvh
    for i, n in enumerate(lens):
        x = data[i]["x"].double()
        y = P.plain_silu(P.plain_short_conv(x, wconv.double()))
        q = (P.plain_unit(y[:, :kd].view(n, kvh, D)) * D ** -0.5).repeat_interleave(rep, dim=1)
        k = P.plain_unit(y[:, kd:2 * kd].view(n, kvh, D)).repeat_interleave(rep, dim=1)
        dec = P.plain_head_decay(data[i]["a"].double(), dtb.double(), a_log.double())
        o, S = P.plain_delta_recurrence(q, k, y[:, 2 * kd:].view(n, heads, Dv), dec, torch.sigmoid(data[i]["beta"].double()))
        assert torch.allclose(torch.cat(got[i]).double(), o.reshape(n, vd), atol=1e-4, rtol=1e-4), \
            (i, float((torch.cat(got[i]).double() - o.reshape(n, vd)).abs().max()))
        assert torch.allclose(state[slots[i], :heads * D * Dv].cpu().double(), S.reshape(-1), atol=1e-4, rtol=1e-4)
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, C, dtype=F64), x])[-(taps - 1):]
            assert torch.equal(state[slots[i], heads * D * Dv:].cpu().double(), tail.reshape(-1)), f"conv tail of request {i}"
    unused = [s for s in range(4) if s not in slots][0]
    assert (state[unused] == 0).all()


@gpu
@pytest.mark.parametrize("portion", [1, 2, 200, 600])
@pytest.mark.parametrize("D,Dv", [(16, 32), (128, 32)])
def test_delta_rule_remembers_a_token_from_far_back(portion, D, Dv):
    """Decays a hair below one and later tokens that write along other keys: what token 0 wrote along its key is still read
    599 tokens on, in single tokens and in portions."""
    from airun_b200.kernels import ops
    n, decay = 600, 0.9995
    q, k, v = torch.zeros(n, D), torch.zeros(n, D), torch.zeros(n, Dv)
    k[0, 3], v[0] = 1.0, torch.arange(Dv) - 10.0
    q[:, 3] = 1.0
    k[1:, 5], v[1:, 0] = 1.0, 1.0
    state = torch.zeros(1, D * Dv, device="cuda")
    qd, kd_, vd, bd = dev(q), dev(k), dev(v), dev(torch.full((n, 1), 30.0))          # sigmoid(30) = 1
    a = dev(torch.full((n, 1), math.log(math.expm1(-math.log(decay)))))              # softplus(a) = -ln(decay)
    one = torch.zeros(1, device="cuda")
    for t in range(0, n, portion):
        ctx = batch_ctx([(t, t + portion)])
        o = torch.empty(portion, Dv, device="cuda")
        s = slice(t, t + portion)
        ops.recurrent_state(ops.RECURRENCE_DELTA_HEAD, qd[s], kd_[s], vd[s], a[s], state, ctx, o, 1, 1, D, Dv, beta=bd[s], a_log=one, dt_bias=one)
    assert torch.allclose(o[-1].cpu().double(), decay ** (n - 1) * v[0].double(), rtol=1e-3, atol=1e-3)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,I,limit", [(33, 100, 24, 0.5), (200, 128, 64, 1.0), (1, 64, 16, 3.0), (300, 256, 96, 0.9)])
def test_clamped_feed_forward(T, H, I, limit, dtype):
    from airun_b200.parts.base import make_part
    g = torch.Generator().manual_seed(T)
    W = {"p.gate": 3 * torch.randn(I, H, generator=g) / math.sqrt(H), "p.up": 3 * torch.randn(I, H, generator=g) / math.sqrt(H),
         "p.down": torch.randn(H, I, generator=g) / math.sqrt(I)}
    W = {n: P.to_bf16_and_back(t) for n, t in W.items()}
    part = make_part("feed_forward", "clamped_glu", prefix="p", hidden_size=H, intermediate_size=I, limit=limit, dtype=dtype, device="cuda")
    part.load_weights({n: dev(t, dtype) for n, t in W.items()})
    h = P.to_bf16_and_back(torch.randn(T, H, generator=g))
    ctx = batch_ctx([(0, T)])
    out = part.forward(ctx, dev(h, dtype))
    rnd = P.to_bf16_and_back if dtype == torch.bfloat16 else None
    want = P.plain_feed_forward(h.double(), W["p.gate"].double(), W["p.up"].double(), W["p.down"].double(), limit, rnd)
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    assert int(ctx.err.item()) == 0 and torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol)


# ----------------------------------------------------------------------------- whole models
@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_whole_prompts_with_the_residual_after_every_layer_run(folders, name, dtype):
    folder, cfg, W, page = folders[name]
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
            assert len(layers) == len(after) == len(P.run_order(cfg))
            for ci in range(len(after)):
                assert np.allclose(layers[ci][:n], after[ci].numpy(), atol=2e-4, rtol=2e-5), (name, ci)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_prompt_then_single_tokens_and_from_the_first_token(folders, name, dtype):
    folder, cfg, W, page = folders[name]
    eng = engine(folder, dtype, page)
    s = random_tokens(97, cfg["vocab"], 3)
    got = run_schedule(eng, [s], [[(0, 40)]] + [[(0, 1)]] * 57)[0]          # the windows and several pages pass over decoded tokens
    compare(got, cfg, W, s, dtype, f"{name} prompt then single tokens")
    s = random_tokens(30, cfg["vocab"], 4)
    got = run_schedule(eng, [s], [[(0, 1)]] * 30)[0]
    compare(got, cfg, W, s, dtype, f"{name} decoded from the first token")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SHAPES))
def test_portions_of_every_size(folders, name, dtype):
    folder, cfg, W, page = folders[name]
    eng = engine(folder, dtype, page)
    s = random_tokens(140, cfg["vocab"], 5)
    for cuts in ([2] * 70, [3, 5, 7, 11, 13, 17, 19, 23, 29, 13], [64, 2, 2, 1, 1, 70], [16, 17, 15, 33, 31, 8, 20]):
        assert sum(cuts) == 140
        got = run_schedule(eng, [s], [[(0, n)] for n in cuts])[0]
        compare(got, cfg, W, s, dtype, f"{name} portions {cuts[:4]}")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["l1", "l2", "l4"])
def test_unequal_requests_through_few_slots_and_pages(folders, name, dtype):
    """Six requests through three slots and a pool that holds about two of them: pages and state slots are freed and
    used again; each request's logits equal the plain ones and those of the request run alone."""
    folder, cfg, W, page = folders[name]
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
def test_long_decoding(folders):
    folder, cfg, W, page = folders["l2"]
    eng = engine(folder, "float32", page, tokens=640)
    s = random_tokens(420, cfg["vocab"], 8)
    got = run_schedule(eng, [s], [[(0, 20)]] + [[(0, 1)]] * 400)[0]
    compare(got, cfg, W, s, "float32", "l2 four hundred single tokens")


ORDERS = {
    "attention only, one pass over the last layer": P.make_config(96, 64, [
        P.attention_layer(2, 1, 16, window=9, rot=8), P.attention_layer(2, 2, 32, rot=16, mlp=P.dense(48, 1.0))], loop=(1, 2, 1)),
    "delta rule only, no feed-forward anywhere, five passes": P.make_config(96, 48, [
        P.delta_layer(2, 1, 8, 24, 2), P.delta_layer(3, 3, 8, 8, 5)], loop=(0, 1, 5), emb_scale=2.0),
    "an empty loop": P.make_config(80, 64, [P.attention_layer(4, 4, 16, window=5, rot=2, mlp=P.dense(32, 2.0)), P.delta_layer(2, 2, 16, 16, 3)],
                                   loop=(1, 1, 3)),
    "a loop that runs no time leaves its layers out": P.make_config(80, 64, [
        P.delta_layer(2, 2, 16, 16, 3), P.attention_layer(4, 4, 16, rot=4), P.delta_layer(1, 1, 8, 16, 2, mlp=P.dense(16, 1.0))], loop=(1, 2, 0)),
}


@gpu
@pytest.mark.parametrize("which", list(ORDERS))
def test_other_orders_of_layers(which, tmp_path):
    cfg = ORDERS[which]
    W = P.random_weights(cfg, seed=len(which))
    folder = P.write_folder(str(tmp_path / "m"), cfg, W)
    s = random_tokens(70, cfg["vocab"], 9)
    for dtype in ("float32", "bfloat16"):
        eng = engine(folder, dtype, 8)
        got = run_schedule(eng, [s], [[(0, 33)], [(0, 2)], [(0, 1)], [(0, 34)]])[0]
        compare(got, cfg, W, s, dtype, which)


@gpu
def test_greedy_generation_through_the_engine(folders):
    """Through the engine's own entry points and scheduler: add_request / run_step for unequal requests at once, and
    generate."""
    import airun_b200
    folder, cfg, W, page = folders["l1"]
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
    folder, cfg, W, page = folders["l2"]
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
