"""GPU tests of the Momedra design on the layer-list path: the CUDA backend (forward / sessions / decode_greedy behind
arch.load_model) against the plain numpy oracle in tests/_momedra_ref.py, on small random models made here.

float32 mode is compared tightly with the oracle; bfloat16 mode loosely with the oracle."""
import json
import os
import subprocess

import numpy as np
import pytest

from powerserve_b200 import arch, arch_synth, capi
from tests import _momedra_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
AT, LA, RG = arch_synth.momedra_attention_layer, arch_synth.momedra_latent_layer, arch_synth.momedra_rglru_layer
# every mixer and feed-forward, a looped pair in the middle, unequal head counts and sizes
MIXED = [LA(3, 8, 6, 10, 20, ff=24, experts=5, top=2, shared_ff=40), AT(4, 2, 10, 14, q_temp=(0.6, 17), ff=56), RG(48, 3, conv=4, ff=16, experts=6, top=3), AT(2, 1, 12, 6, q_temp=(0.3, 50))]
MIXED_LOOP = (1, 3, 3)


def make(tmp_path, layers, width=48, vocab=96, seed=0, eps=1e-5, edit=None, name="m", loop=None, residual_mult=0.6):
    cfg = arch_synth.momedra_config(width, vocab, layers, loop=loop, eps=eps, residual_mult=residual_mult)
    t = arch_synth.momedra_weights(cfg, seed=seed)
    if edit:
        edit(t)
        t = {k: R.bf16_round(v) for k, v in t.items()}
    d = str(tmp_path / name)
    arch_synth.write_model_dir(d, cfg, t)
    return d, cfg, t


def tokens(vocab, n, seed=0):
    return [int(v) for v in np.random.default_rng(seed).integers(0, vocab, n)]


def run(model, toks, cuts=None):
    """logits of every position, the sequence fed in portions of the given sizes (cycled); None = one portion per batch cap"""
    model.reset()
    cap, out, lo, k = model.desc.max_batch, [], 0, 0
    while lo < len(toks):
        s = min(cap if cuts is None else min(cuts[k % len(cuts)], cap), len(toks) - lo)
        out.append(model.forward(toks[lo:lo + s]))
        lo, k = lo + s, k + 1
    return np.concatenate(out)


def rel_err(got, ref):
    """per position: rms of the difference over rms of the reference"""
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.maximum(np.sqrt((ref ** 2).mean(-1)), 1e-6)


TOL = {"float32": 4e-5, "bfloat16": 6e-2}


def check(got, ref, dtype, what=""):
    e = rel_err(got, ref)
    assert e.max() < TOL[dtype], f"{what}: worst relative error {e.max():.3g} at position {int(e.argmax())} ({dtype})"
    if dtype == "bfloat16":
        assert np.median(e) < 2e-2, f"{what}: median relative error {np.median(e):.3g}"


def check_routed_bf16(got, ref, what=""):
    """models with a router: a position whose choice is a close call may flip under rounding, so a few positions may be far off"""
    e = rel_err(got, ref)
    assert np.median(e) < 2e-2 and np.mean(e > TOL["bfloat16"]) < 0.1, f"{what}: median {np.median(e):.3g}, {np.mean(e > TOL['bfloat16']):.3g} of the positions over"


def both_paths(d, toks, ref, what, n_ctx, cap=64, cuts=([7, 2, 33, 1],), decode_from=None):
    """float32: portions of the batch cap, ragged portions, and the tail decoded token by token, all against the oracle"""
    m = arch.load_model(d, dtype="float32", max_batch=cap, n_ctx=n_ctx)
    check(run(m, toks), ref, "float32", what + ", portions of the batch cap")
    for c in cuts:
        check(run(m, toks, list(c)), ref, "float32", what + f", portions {list(c)}")
    k = decode_from if decode_from is not None else len(toks) // 2
    m.reset()
    for lo in range(0, k, cap):
        m.forward(toks[lo:min(k, lo + cap)], lm_head=False)
    dec = np.concatenate([m.forward(toks[i:i + 1]) for i in range(k, len(toks))])
    check(dec, ref[k:], "float32", what + ", decoded alone")
    m.close()


def alone(tmp_path, layer, what, seed, n=45, width=48, n_ctx=64, moved=(), **kw):
    """one layer by itself, its residual stream too; `moved`: (tensor, value) pairs that must show in the oracle's logits"""
    d, cfg, t = make(tmp_path, [layer], seed=seed, width=width, **kw)
    toks = tokens(96, n, seed)
    taps = []
    ref = R.forward(cfg, t, toks, taps=taps)
    for name, new in moved:
        t2 = dict(t)
        t2[name] = np.full_like(t[name], new)
        assert rel_err(R.forward(cfg, t2, toks), ref).max() > 5e-3, name
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=n_ctx)
    m.be.set_option("arch_taps", 1)
    check(run(m, toks), ref, "float32", what)
    check(m.layer_tap(0, len(toks)), taps[0], "float32", "residual after the layer")
    m.close()
    both_paths(d, toks, ref, what, n_ctx, cuts=([7, 2, 33, 1], [2]))


# ------------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,q_temp", [(4, 2, 10, 14, (0.5, 7)), (3, 3, 8, 8, (1.5, 1)), (6, 1, 12, 4, (0.25, 44)), (1, 1, 6, 20, None), (8, 4, 16, 16, (0.8, 16))])
def test_attention_layer_alone(tmp_path, heads, kv_heads, dim, vdim, q_temp):
    alone(tmp_path, AT(heads, kv_heads, dim, vdim, q_temp=q_temp), "attention-only layer", 1,
          moved=[("l0.mix.g", 0.0), ("l0.mix.q.norm", 1.0), ("l0.mix.k.norm", 0.5), ("l0.mix.q.b", 0.0), ("l0.mix.v.b", 0.0)])


@pytest.mark.parametrize("geometry", [(3, 8, 6, 10, 20), (2, 4, 8, 4, 9), (1, 6, 2, 5, 7), (4, 16, 16, 12, 24), (5, 24, 8, 40, 72), (9, 8, 4, 8, 16)])
def test_latent_layer_alone(tmp_path, geometry):
    alone(tmp_path, LA(*geometry, rope_base=500.0), "latent attention with a sink", 3, moved=[("l0.mix.sink", -30.0), ("l0.mix.dkv.norm", 0.5)])


@pytest.mark.parametrize("width,blocks,conv", [(24, 3, 4), (7, 1, 2), (64, 4, 1), (30, 30, 3), (72, 2, 7), (256, 2, 4)])
def test_rglru_layer_alone(tmp_path, width, blocks, conv):
    alone(tmp_path, RG(width, blocks, conv=conv), "gated linear recurrence", 4, n_ctx=48, moved=[("l0.mix.ra.b", 3.0), ("l0.mix.ri.b", 3.0), ("l0.mix.lam", -4.0), ("l0.mix.y.b", 1.0), ("l0.mix.conv.b", 1.0)])


@pytest.mark.parametrize("lam", [-20.0, -9.0, 0.0, 4.0])
def test_decays_from_nearly_one_to_nearly_zero(tmp_path, lam):
    """1 - a^2 must not cancel when a is close to one: the float64 oracle shows it"""
    def edit(t):
        t["l0.mix.lam"] = np.full_like(t["l0.mix.lam"], lam)
        t["l0.mix.o"] = t["l0.mix.o"] * np.float32({-20.0: 512.0, -9.0: 16.0}.get(lam, 1.0))
    alone(tmp_path, RG(32, 2, conv=3), f"lam = {lam}", 5, n=48, n_ctx=48, edit=edit)


def test_dense_feed_forward_alone(tmp_path):
    alone(tmp_path, RG(4, 1, conv=1, ff=72), "feed-forward without a gate", 6, moved=[("l0.mlp.up", 0.0)])


@pytest.mark.parametrize("experts,top,ff,shared", [(5, 2, 24, 40), (16, 3, 20, 12), (3, 3, 17, 9), (1, 1, 8, 0), (40, 5, 12, 0), (130, 4, 8, 16)])
def test_routed_feed_forward_alone(tmp_path, experts, top, ff, shared):
    alone(tmp_path, RG(4, 1, conv=1, ff=ff, experts=experts, top=top, shared_ff=shared), "routed experts", 7,
          moved=([("l0.mlp.shared.down", 0.0)] if shared else []) + ([("l0.mlp.router.b", 0.0)] if top < experts else []))


def test_residual_factor(tmp_path):
    for mult in (1.0, 0.25, 1.6):
        layers = [AT(2, 1, 8, 8, ff=16), RG(12, 2)]
        d, cfg, t = make(tmp_path, layers, seed=8, residual_mult=mult, name=f"m{mult}")
        toks = tokens(96, 30, 8)
        both_paths(d, toks, R.forward(cfg, t, toks), f"residual factor {mult}", 32, cap=16)


# ------------------------------------------------------------------------------------------------- far keys, edges, the start
def find_far(layer_edit, layer, tmp_path, seed, n=340, at=27, ask=(297, 320, 339), **kw):
    """a token that occurs once, far back; the token that asks for it has the opposite embedding and the layer's queries are minus its keys,
    so that the far key matches and the asking token's own key does not"""
    d, cfg, t = make(tmp_path, [layer], seed=seed, width=32, vocab=40, edit=layer_edit, **kw)
    toks = [1 + int(v) for v in np.random.default_rng(seed).integers(0, 38, n)]
    toks[at] = 0
    for p in ask:
        toks[p] = 39
    ref = R.forward(cfg, t, toks)
    other = list(toks)
    other[at] = 5
    assert rel_err(R.forward(cfg, t, other)[list(ask)], ref[list(ask)]).min() > 2e-2   # the far token matters where it is asked for
    both_paths(d, toks, ref, "far token", -(-n // 16) * 16, cap=128, cuts=([100, 3, 128], [64]), decode_from=ask[0] - 2)
    return d, toks, ref


@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 127, 255])
def test_a_far_key_of_the_attention(tmp_path, at):
    """one head whose query is minus its key: at the borders of the kernels' 16-key blocks and 64-key tiles, and the first token"""
    def edit(t):
        t["l0.mix.q"] = -t["l0.mix.k"]
        t["l0.mix.q.b"], t["l0.mix.k.b"] = t["l0.mix.q.b"] * 0, t["l0.mix.k.b"] * 0
        t["l0.mix.q.norm"] = t["l0.mix.q.norm"] * 3.0
        t["embed"][39] = -t["embed"][0]
    find_far(edit, AT(1, 1, 16, 8, q_temp=(0.7, 64), scale=1.0), tmp_path, 9, at=at)


@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 127, 255])
def test_a_far_latent(tmp_path, at):
    """the plain part of the query is minus the latent; the rotated part is turned down so that distance does not hide the match"""
    def edit(t):
        dn, rk = 16, 16
        t["l0.mix.uk"] = np.eye(dn, rk, dtype=np.float32)
        q = np.zeros_like(t["l0.mix.q"])
        q[:dn] = -4.0 * t["l0.mix.dkv"][:rk]
        q[dn:] = 0.05 * t["l0.mix.q"][dn:]
        t["l0.mix.q"] = q
        t["l0.mix.dkv.norm"] = np.ones_like(t["l0.mix.dkv.norm"])
        t["embed"][39] = -t["embed"][0]
    find_far(edit, LA(1, 16, 4, 8, 16, scale=1.0), tmp_path, 10, at=at)


def test_position_alone_moves_the_query_temperature(tmp_path):
    """`every` at the kernels' block and tile borders, and off by one it shows in the oracle by far more than the tolerance"""
    for every in (1, 15, 16, 64, 100):
        def edit(t):
            t["l0.mix.q.norm"] = t["l0.mix.q.norm"] * 2.0
        d, cfg, t = make(tmp_path, [AT(2, 1, 8, 8, q_temp=(1.3, every))], seed=11, width=32, name=f"e{every}", edit=edit)
        toks = tokens(96, 140, 11)
        ref = R.forward(cfg, t, toks)
        c2 = json.loads(json.dumps(cfg))
        c2["layers"][0]["mixer"]["q_temp"]["every"] = every + 1
        e = rel_err(R.forward(c2, t, toks), ref)
        assert e[every - 1] > 1e-2 or every == 1 or every > 140, e[every - 1]
        assert e[:max(every - 1, 0)].max(initial=0.0) < 1e-12
        both_paths(d, toks, ref, f"temperature every {every}", 144, cap=80, cuts=([64, 16, 1],), decode_from=every - 1 if every < 100 else 90)


def test_rotation_far_from_the_start(tmp_path):
    """a base that leaves every pair turning fast: the angle's error would show first at the last positions"""
    def edit(t):
        t["l0.mix.q"] = t["l0.mix.q"] * 3.0
    d, cfg, t = make(tmp_path, [LA(2, 4, 16, 8, 12, rope_base=3.0)], seed=12, width=32, edit=edit)
    toks = tokens(96, 900, 12)
    ref = R.forward(cfg, t, toks)
    both_paths(d, toks, ref, "rotation", 912, cap=256, cuts=([200, 3],), decode_from=880)


def test_state_reaches_across_portions(tmp_path):
    """slow decays: the first token still shows in the last logits, through every cut"""
    def edit(t):
        t["l0.mix.lam"] = np.full_like(t["l0.mix.lam"], -9.0)
        t["l0.mix.o"] = t["l0.mix.o"] * 8.0
        t["embed"][0] = t["embed"][0] * 0 + 8.0 * np.sign(t["embed"][1])
    d, cfg, t = make(tmp_path, [RG(32, 2, conv=5)], seed=13, width=32, edit=edit)
    toks = [0] + [1 + v % 95 for v in tokens(95, 199, 13)]
    ref = R.forward(cfg, t, toks)
    assert rel_err(R.forward(cfg, t, [7] + toks[1:])[-1:], ref[-1:]).max() > 1e-3
    both_paths(d, toks, ref, "state", 208, cap=96, cuts=([2], [3, 1, 4], [32], [33, 31]), decode_from=40)


def test_the_first_tokens(tmp_path):
    """the first tokens of a sequence on a set that a longer sequence has used: nothing of it may show (keys, state, convolution inputs)"""
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=14, loop=MIXED_LOOP)
    long_, short = tokens(130, 60, 14), tokens(130, 6, 15)
    ref = R.forward(cfg, t, short)
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=64)
    for cuts in ([1], [2], [6], [3, 1]):
        run(m, long_)
        check(run(m, short, cuts), ref, "float32", f"first tokens, portions {cuts}")
    m.close()


# ------------------------------------------------------------------------------------------------- passes
@pytest.mark.parametrize("loop", [(0, 2, 3), (1, 3, 2), (0, 1, 1), (2, 3, 4), (0, 3, 2), None])
def test_looped_runs(tmp_path, loop):
    """every run's residual stream against the oracle's: shared weights, a cache and state per run, the embedding output projected in"""
    layers = [AT(2, 2, 8, 6, ff=24), RG(20, 2, conv=3, ff=12, experts=4, top=2, shared_ff=8), LA(2, 6, 4, 6, 10, ff=16)]
    d, cfg, t = make(tmp_path, layers, seed=16, loop=loop, width=40)
    toks = tokens(96, 37, 16)
    taps = []
    ref = R.forward(cfg, t, toks, taps=taps)
    assert len(taps) == (3 if not loop else 3 + (loop[1] - loop[0]) * (loop[2] - 1))
    m = arch.load_model(d, dtype="float32", max_batch=64, n_ctx=48)
    m.be.set_option("arch_taps", 1)
    check(run(m, toks), ref, "float32", f"loop {loop}")
    for i, tap in enumerate(taps):
        check(m.layer_tap(i, len(toks)), tap, "float32", f"residual after run {i}")
    m.close()
    both_paths(d, toks, ref, f"loop {loop}", 48, cap=16, cuts=([5, 2, 16], [2]))


# ------------------------------------------------------------------------------------------------- schedules
def test_whole_prompt_portions_and_decoding_agree_in_both_precisions(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=17, loop=MIXED_LOOP)
    toks = tokens(130, 150, 17)
    ref = R.forward(cfg, t, toks)
    both_paths(d, toks, ref, "mixed model", 160, cap=64, cuts=([7, 2, 33, 1], [2], [64, 3]))
    m = arch.load_model(d, dtype="bfloat16", max_batch=64, n_ctx=160)
    whole = run(m, toks)
    check_routed_bf16(whole, ref, "whole prompt")
    for cuts in ([1], [2], [5, 40, 3]):
        got = run(m, toks, cuts)
        check_routed_bf16(got, ref, f"portions {cuts}")
        assert np.median(rel_err(got, whole)) < 2e-2
    m.close()


def test_bfloat16_without_a_router(tmp_path):
    layers = [AT(4, 2, 16, 8, q_temp=(0.5, 30), ff=64), RG(64, 4, conv=4, ff=64), LA(4, 16, 8, 16, 24, ff=64)]
    d, cfg, t = make(tmp_path, layers, width=64, vocab=120, seed=18, loop=(0, 2, 2))
    toks = tokens(120, 150, 18)
    ref = R.forward(cfg, t, toks)
    m = arch.load_model(d, dtype="bfloat16", max_batch=64, n_ctx=160)
    for cuts in (None, [1], [2, 50]):
        check(run(m, toks, cuts), ref, "bfloat16", f"portions {cuts}")
    m.close()


def test_single_token_kernels_match_the_batch_kernels(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=19, loop=MIXED_LOOP)
    toks = tokens(130, 100, 19)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=32, n_ctx=112)
        a = run(m, toks, [1])
        m.be.set_option("arch_simple", 1)
        b = run(m, toks, [1])
        assert np.median(rel_err(a, b)) < (1e-5 if dtype == "float32" else 2e-2), dtype
        if dtype == "float32":
            assert rel_err(a, b).max() < 8e-5
        m.close()


def test_replayed_step_matches_the_plain_launches(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=20, loop=MIXED_LOOP)
    toks = tokens(130, 90, 20)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=40, n_ctx=96)
        g0 = m.be.counter("graph_replays")
        a = run(m, toks, [1])
        assert m.be.counter("graph_replays") - g0 == len(toks)
        m.reset()
        m.forward(toks[:40], lm_head=False)
        ids_a = list(m.decode_greedy(toks[40], 20))
        m.be.set_option("graph", 0)
        b = run(m, toks, [1])
        m.reset()
        m.forward(toks[:40], lm_head=False)
        ids_b = list(m.decode_greedy(toks[40], 20))
        np.testing.assert_array_equal(a, b)                         # the same kernels on the same data
        assert ids_a == ids_b
        m.be.set_option("graph", 1)
        for opt in ("arch_pdl", "arch_fork"):
            m.be.set_option(opt, 0)
            np.testing.assert_array_equal(run(m, toks, [1]), a)
            m.be.set_option(opt, 1)
        m.close()


def test_tensor_core_gemm_matches_the_tile_kernels(tmp_path):
    """bfloat16 batches: the tcgen05 GEMM (row ranges with and without the activation, concatenated output product, experts without a
    gate, the pass projection) against the fp32-FMA tiles"""
    layers = [AT(6, 3, 24, 40, q_temp=(0.4, 90), ff=200), RG(150, 3, conv=4, ff=136), LA(4, 24, 16, 20, 40, ff=72)]
    d, cfg, t = make(tmp_path, layers, width=136, vocab=300, seed=21, loop=(0, 2, 2))
    toks = tokens(300, 300, 21)
    m = arch.load_model(d, dtype="bfloat16", max_batch=160, n_ctx=304)
    n0 = m.be.counter("kernel_launches")
    a = run(m, toks)
    n1 = m.be.counter("kernel_launches")
    m.be.set_option("arch_tc", 0)
    b = run(m, toks)
    n2 = m.be.counter("kernel_launches")
    assert n1 - n0 > n2 - n1                                        # the tensor-core path adds its operand-tiling launches: it did run
    e = rel_err(a, b)
    assert np.median(e) < 1e-2 and e.max() < 4e-2, (np.median(e), e.max())
    check(a, R.forward(cfg, t, toks), "bfloat16", "tensor-core path against the oracle")
    m.close()
    layers = [AT(6, 3, 24, 40, ff=200, experts=7, top=3, shared_ff=130)]
    d, cfg, t = make(tmp_path, layers, width=136, vocab=300, seed=22, name="moe")
    m = arch.load_model(d, dtype="bfloat16", max_batch=160, n_ctx=304)
    a = run(m, toks)
    m.be.set_option("arch_tc", 0)
    b = run(m, toks)
    e = rel_err(a, b)
    assert np.median(e) < 1e-2 and np.mean(e > 4e-2) < 0.02, (np.median(e), e.max())
    check_routed_bf16(a, R.forward(cfg, t, toks), "experts on the tensor cores")
    m.close()


def test_sessions_interleaved_and_sets_reused(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=23, loop=MIXED_LOOP)
    reqs = [tokens(130, n, 40 + i) for i, n in enumerate((50, 9, 33, 64))]
    refs = [R.forward(cfg, t, r) for r in reqs]
    m = arch.load_model(d, dtype="float32", max_batch=16, n_ctx=64)
    sid = [m.session_create() for _ in range(3)]
    got = [[] for _ in reqs]
    at = [0, 0, 0, 0]
    sizes = [5, 2, 16, 1, 7]
    live, k = [0, 1, 2], 0
    while live:
        for r in list(live):
            s = min(sizes[k % len(sizes)], len(reqs[r]) - at[r])
            k += 1
            m.session_select(sid[r])
            assert m.position == at[r]
            got[r].append(m.forward(reqs[r][at[r]:at[r] + s]))
            at[r] += s
            if at[r] == len(reqs[r]):
                live.remove(r)
                if r == 1:              # the short request ends first: its set is freed and a new request takes a new one
                    m.session_select(0)
                    m.session_destroy(sid[1])
                    sid.append(m.session_create())
                    live.append(3)
    for r in range(4):
        check(np.concatenate(got[r]), refs[r], "float32", f"request {r} among others")
    # the same set used again from position 0: the recurrent state of the longer request must not leak
    m.session_select(sid[0])
    m.reset()
    check(run(m, reqs[2], [16]), refs[2], "float32", "set reused after reset")
    check(run(m, reqs[1], [1]), refs[1], "float32", "set reused once more, token by token")
    m.reset()
    m.forward(reqs[2][:16])
    with pytest.raises(capi.PsCudaError):                           # recurrent state cannot be cut back, only to the start
        m.be.kv_rollback(13)
    m.be.kv_rollback(16)
    assert m.position == 0
    check(m.forward(reqs[2][:16]), refs[2][:16], "float32", "from the start after a rollback to 0")
    m.close()


def test_long_decoding(tmp_path):
    layers = [AT(4, 1, 8, 12, q_temp=(0.5, 60), ff=16), RG(24, 2, conv=4, ff=16, experts=4, top=2), LA(2, 8, 4, 6, 12, ff=8)]
    d, cfg, t = make(tmp_path, layers, width=32, vocab=50, seed=24, loop=(0, 2, 2))
    toks = tokens(50, 400, 24)
    ref = R.forward(cfg, t, toks)
    for dtype in ("float32", "bfloat16"):
        m = arch.load_model(d, dtype=dtype, max_batch=8, n_ctx=400)
        m.reset()
        m.forward(toks[:6], lm_head=False)
        dec = np.concatenate([m.forward(toks[i:i + 1]) for i in range(6, 400)])
        if dtype == "float32":
            check(dec, ref[6:], dtype, "394 tokens decoded alone")
        else:
            check_routed_bf16(dec, ref[6:], "394 tokens decoded alone")
        m.close()


@pytest.mark.parametrize("layers,width,vocab,loop", [
    ([AT(1, 1, 1, 1, q_temp=(0.5, 2))], 8, 11, None),                                               # the smallest of everything
    ([RG(1, 1, conv=1, ff=1)], 8, 11, (0, 1, 2)),
    ([LA(1, 4, 2, 1, 1, ff=3)], 8, 11, None),
    ([AT(8, 8, 8, 8, ff=8)], 40, 64, None),                                                         # no key sharing
    ([AT(12, 1, 12, 20, ff=20, experts=2, top=1, shared_ff=7)], 56, 77, (0, 1, 3)),                 # one shared key head
    ([RG(35, 7, conv=5, ff=37), LA(3, 5, 6, 7, 11, ff=13), AT(5, 5, 7, 9, ff=11, experts=3, top=2)], 50, 101, (1, 3, 2)),   # nothing a multiple of four
    ([LA(16, 32, 16, 24, 48, ff=96), AT(16, 4, 32, 64, ff=96, experts=8, top=2, shared_ff=64), RG(256, 4, conv=4, ff=96)], 128, 300, (0, 3, 2)),
    ([RG(640, 2, conv=4), RG(96, 96, conv=2)], 96, 60, (0, 2, 1)),                                  # wide blocks; blocks of one channel
    ([AT(2, 2, 8, 8), AT(4, 1, 8, 4), LA(2, 8, 4, 8, 8)], 32, 60, None),                            # no feed-forward anywhere
])
def test_other_sizes(tmp_path, layers, width, vocab, loop):
    d, cfg, t = make(tmp_path, layers, width=width, vocab=vocab, seed=25, eps=3e-6, loop=loop, residual_mult=0.9)
    toks = tokens(vocab, 75, 25)
    ref = R.forward(cfg, t, toks)
    m = arch.load_model(d, dtype="float32", max_batch=32, n_ctx=80)
    check(run(m, toks), ref, "float32", "portions of 32")
    check(run(m, toks, [2, 31, 1]), ref, "float32", "ragged portions")
    check(run(m, toks[:40], [1]), ref[:40], "float32", "token by token")
    m.close()
    m = arch.load_model(d, dtype="bfloat16", max_batch=80, n_ctx=80)
    check_routed_bf16(run(m, toks), ref, "whole prompt")
    m.close()


# ------------------------------------------------------------------------------------------------- entry points
def test_greedy_generation_through_the_entry_points(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=26, loop=MIXED_LOOP)
    prompt = tokens(130, 21, 26)
    m = arch.load_model(d, dtype="float32", max_batch=8, n_ctx=64)
    ids, lg = m.generate(prompt, 12, batch_size=8)                  # prefill in portions + one forward per token
    m.reset()
    m.prefill(prompt, 8)
    ids2 = [int(v) for v in m.decode_greedy(prompt[-1], 12)]        # the device-side greedy loop
    assert ids == ids2
    assert m.position == len(prompt) - 1 + 12
    seq = list(prompt)
    for step, tok in enumerate(ids):
        ref = R.forward(cfg, t, seq)[-1]
        assert rel_err(lg[step][None], ref[None]).max() < 4e-5
        assert ref[tok] >= ref.max() - 1e-4 * np.abs(ref).max()
        seq.append(tok)
    m.forward_lazy([seq[-1]])
    vals, idx = m.sample_topk(5)
    full = R.forward(cfg, t, seq)[-1]
    assert list(idx) == [int(v) for v in np.argsort(-full, kind="stable")[:5]]
    m.close()


def test_bad_configurations_are_refused(tmp_path):
    odd = LA(2, 8, 5, 4, 6)                                          # an odd number of rotated dimensions
    for i, layers in enumerate([[AT(3, 2, 8, 8)], [RG(10, 3)], [odd], [RG(8, 1, ff=8, experts=2, top=3)]]):
        with pytest.raises((capi.PsCudaError, KeyError)):
            cfg = arch_synth.momedra_config(32, 40, layers)
            t = arch_synth.momedra_weights(arch_synth.momedra_config(32, 40, [AT(2, 1, 8, 8)]), seed=27)
            arch_synth.write_model_dir(str(tmp_path / f"bad{i}"), cfg, t)
            arch.load_model(str(tmp_path / f"bad{i}"), dtype="float32", max_batch=8, n_ctx=16)


def test_trace_runner_and_generation_command_lines(tmp_path):
    d, cfg, t = make(tmp_path, MIXED, width=72, vocab=130, seed=28, loop=MIXED_LOOP)
    a, b = tokens(130, 40, 30), tokens(130, 17, 31)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[32:], "want": [7, 3]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [16]}], "end": ["b"]}]
    out = tmp_path / "out"
    ra, rb = R.forward(cfg, t, a), R.forward(cfg, t, b)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "40", "--max-batch", "16"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    check(np.fromfile(out / "0.f32", "<f4").reshape(2, 130), ra[[0, 29]], "float32", "step 0")
    assert not (out / "1.f32").exists()
    check(np.fromfile(out / "2.f32", "<f4").reshape(2, 130), ra[[39, 35]], "float32", "step 2 (order of `want`)")
    check(np.fromfile(out / "3.f32", "<f4").reshape(1, 130), rb[[16]], "float32", "step 3")
    prompt = tokens(130, 19, 29)
    exe = os.path.join(ROOT, "bin", "ps_generate")
    p = subprocess.run([exe, "--model", d, "--dtype", "float32", "--ids", " ".join(map(str, prompt)), "--n", "10", "--prefill-batch", "8"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = json.loads(p.stdout.strip().splitlines()[-1])["ids"]
    m = arch.load_model(d, dtype="float32", max_batch=32, n_ctx=32)
    want, _ = m.generate(prompt, 10, batch_size=8)
    assert ids == want
    m.close()
