"""CPU-only checks around the Momedra design: the registry's reading of a configuration (every size and constant comes from the
file, a looped group of layers becomes runs that share weights), the tensor names, and the oracle's own invariants (it is what
the GPU tests compare with, so it is checked against hand-computed cases and second formulations here)."""
import math

import numpy as np
import pytest

from powerserve_b200 import arch, arch_synth, capi
from tests import _momedra_ref as R

AT, LA, RG = arch_synth.momedra_attention_layer, arch_synth.momedra_latent_layer, arch_synth.momedra_rglru_layer
DESCRIBE, NAMES = arch.ARCHITECTURES["Momedra"]


def test_registry_reads_every_size_from_the_configuration():
    layers = [LA(5, 12, 6, 9, 21, scale=0.19, rope_base=1234.0, ff=44), AT(6, 3, 10, 14, scale=0.21, q_temp=(0.7, 33), ff=18, experts=11, top=4, shared_ff=26),
              RG(55, 5, conv=6, ff=12), AT(2, 2, 7, 5, q_temp=None), RG(8, 1, conv=1, ff=9, experts=3, top=3)]
    cfg = arch_synth.momedra_config(60, 99, layers, loop=(1, 3, 2), eps=3e-5, residual_mult=0.35)
    descs, top = DESCRIBE(cfg, {})
    assert top == {"dim": 60, "vocab_size": 99, "norm_eps": 3e-5, "embed_scale": 1.0, "norm_unit_offset": 0, "norm_kind": capi.NORM_LAYER, "residual_scale": 0.35}
    assert len(descs) == 7                                           # latent, (attention, rg-lru) twice, attention, rg-lru
    assert all(d.block_kind == capi.BLOCK_PARALLEL and d.post_norm == 0 and d.raw_input == 0 and d.window == 0 for d in descs)
    d = descs[0]
    assert (d.mixer_kind, d.n_heads, d.n_kv_heads, d.qk_dim, d.rot_dim, d.v_dim, d.q_rank, d.kv_rank) == (capi.MIXER_LATENT, 5, 1, 12, 6, 9, 0, 21)
    assert (d.rope_dims, d.rope_base, d.rope_interleaved, d.rope_factor, d.sink) == (6, 1234.0, 1, 0.0, capi.SINK_LEARNED) and abs(d.score_scale - 0.19) < 1e-7
    assert (d.mlp_kind, d.expert_ff, d.mlp_ungated, d.act_kind, d.proj_bias, d.out_gate, d.qk_norm) == (capi.MLP_DENSE, 44, 1, capi.ACT_RELU2, 0, 0, 0)
    assert (d.share_weights, d.pass_in) == (0, 0)
    d = descs[1]
    assert (d.mixer_kind, d.n_heads, d.n_kv_heads, d.qk_dim, d.v_dim, d.proj_bias, d.qk_norm, d.out_gate) == (capi.MIXER_ATTENTION, 6, 3, 10, 14, 2, capi.QKNORM_HEAD_W, capi.GATE_HEAD)
    assert abs(d.score_scale - 0.21) < 1e-7 and abs(d.q_temp_coef - 0.7) < 1e-7 and d.q_temp_every == 33.0 and d.sink == capi.SINK_NONE
    assert (d.mlp_kind, d.n_experts, d.top_k, d.expert_ff, d.shared_ff, d.shared_gate, d.router_act, d.router_bias, d.route_on_input) == \
        (capi.MLP_ROUTED, 11, 4, 18, 26, 0, capi.ROUTER_TOPK_SOFTMAX, 1, 0)
    assert (d.share_weights, d.pass_in) == (0, 1)                    # the first pass projects the embedding output in as well
    d = descs[2]
    assert (d.mixer_kind, d.rec_width, d.rec_blocks, d.conv_taps, d.rec_rate, d.expert_ff) == (capi.MIXER_RGLRU, 55, 5, 6, 8.0, 12)
    assert (d.share_weights, d.pass_in) == (0, 0)
    assert (descs[3].share_weights, descs[3].pass_in, descs[4].share_weights, descs[4].pass_in) == (2, 1, 3, 0)
    assert (descs[5].mlp_kind, descs[5].q_temp_coef, descs[5].pass_in) == (capi.MLP_NONE, 0.0, 0)
    assert (descs[6].conv_taps, descs[6].shared_ff, descs[6].top_k) == (1, 0, 3)


@pytest.mark.parametrize("loop,want", [((0, 2, 3), [0, 1, 0, 1, 0, 1, 2]), ((1, 3, 2), [0, 1, 2, 1, 2]), ((0, 1, 1), [0, 1, 2]), (None, [0, 1, 2]), ((1, 1, 5), [0, 1, 2])])
def test_runs_follow_the_loop(loop, want):
    cfg = arch_synth.momedra_config(16, 8, [RG(4, 1)] * 3, loop=loop)
    assert [i for i, _ in R.layer_runs(cfg)] == want
    descs, _ = DESCRIBE(cfg, {})
    assert [bool(d.pass_in) for d in descs] == [o for _, o in R.layer_runs(cfg)]
    assert sum(d.pass_in for d in descs) == (loop[2] if loop and loop[1] > loop[0] else 0)
    names = NAMES(cfg)
    assert ("pass_in" in names) == bool(loop and loop[1] > loop[0])
    assert [n == {} for n in names["layers"]] == [d.share_weights > 0 for d in descs]


def test_bad_types_are_refused():
    cfg = arch_synth.momedra_config(16, 8, [AT(1, 1, 4, 4)])
    cfg["layers"][0]["type"] = "retention"
    with pytest.raises(capi.PsCudaError):
        DESCRIBE(cfg, {})
    cfg = arch_synth.momedra_config(16, 8, [AT(1, 1, 4, 4, ff=8)])
    cfg["layers"][0]["mlp"]["kind"] = "gated"
    with pytest.raises(capi.PsCudaError):
        DESCRIBE(cfg, {})
    with pytest.raises(capi.PsCudaError):
        DESCRIBE(arch_synth.momedra_config(16, 8, [RG(4, 1)], loop=(0, 2, 1)), {})


def test_tensor_names_follow_the_layer_types():
    cfg = arch_synth.momedra_config(16, 8, [AT(2, 1, 4, 6, ff=8, experts=3, top=2, shared_ff=5), RG(12, 3, ff=8), LA(2, 4, 2, 4, 5), RG(4, 1, ff=4, experts=2)], loop=(0, 2, 2))
    n = NAMES(cfg)
    t = arch_synth.momedra_weights(cfg, seed=1)
    used = {n["embed"], n["final_norm"], n["head"], n["pass_in"]}
    for ln in n["layers"]:
        for v in ln.values():
            used.update(v if isinstance(v, list) else [v])
    assert used == set(t)                                            # every stored tensor is named once, nothing else is
    assert t["loop.in"].shape == (16, 32) and t["l1.mix.ra"].shape == (3, 4, 4) and t["l1.mix.ra.b"].shape == (3, 4) and t["l0.mix.g"].shape == (2, 16)
    assert t["l2.mix.dkv"].shape == (7, 16) and t["l2.mix.q"].shape == (12, 16) and t["l0.mlp.shared.up"].shape == (5, 16) and "l3.mlp.shared.up" not in t


# ------------------------------------------------------------------------------------------------- the oracle by hand
def test_small_functions_by_hand():
    assert R.relu_squared(np.array([-2.0, 0.0, 3.0])).tolist() == [0.0, 0.0, 9.0]
    z = 0.7
    assert abs(float(R.gelu_tanh(np.array(z))) - 0.5 * z * (1 + math.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))) < 1e-15
    x, w = np.array([[1.0, 2.0, 3.0, 6.0]]), np.array([1.0, 2.0, 0.5, -1.0])
    np.testing.assert_allclose(R.layer_norm(x, w, 0.25), (x - 3.0) / math.sqrt(14 / 4 + 0.25) * w)
    np.testing.assert_allclose(R.rms_norm(x, w, 0.5), x / math.sqrt(50 / 4 + 0.5) * w)


def test_query_temperature_steps_at_every_multiple():
    t = {"coef": 0.5, "every": 4}
    got = R.query_temperature(np.arange(12), t)
    want = [1.0 + 0.5 * math.log(1 + n) for n in (0, 0, 0, 1, 1, 1, 1, 2, 2, 2, 2, 3)]      # floor((p + 1) / 4)
    np.testing.assert_allclose(got, want)
    assert R.query_temperature([5, 6], None).tolist() == [1.0, 1.0]


def test_sink_only_widens_the_denominator():
    s = np.array([[0.0, 9.0], [1.0, 2.0]])
    p = R.causal_softmax(s, 0.5)
    np.testing.assert_allclose(p, [[1 / (1 + math.exp(0.5)), 0.0], [math.e / (math.e + math.exp(2) + math.exp(0.5)), math.exp(2) / (math.e + math.exp(2) + math.exp(0.5))]])
    np.testing.assert_allclose(R.causal_softmax(s).sum(-1), 1.0)
    np.testing.assert_allclose(R.causal_softmax(s, -1e9), R.causal_softmax(s))
    assert R.causal_softmax(s, 50.0).max() < 1e-18


def test_rotation_in_neighbouring_pairs():
    v = np.arange(1.0, 7.0)[None, :]
    out = R.rotate_pairs(v, [3], 6, 100.0)
    for i in range(3):
        a = 3 * 100.0 ** (-2.0 * i / 6)
        u, w = v[0, 2 * i], v[0, 2 * i + 1]
        np.testing.assert_allclose(out[0, 2 * i:2 * i + 2], [u * math.cos(a) - w * math.sin(a), w * math.cos(a) + u * math.sin(a)])


def test_routing_by_hand():
    w = R.route(np.array([[0.0, 2.0, -1.0, 1.0]]), 2)
    e = math.exp(-1.0)
    np.testing.assert_allclose(w, [[0, 1 / (1 + e), 0, e / (1 + e)]])
    np.testing.assert_allclose(R.route(np.array([[3.0, 1.0]]), 1), [[1.0, 0.0]])
    np.testing.assert_allclose(R.route(np.array([[3.0, 1.0]]), 2).sum(), 1.0)


def test_convolution_and_recurrence_against_explicit_loops():
    rng = np.random.default_rng(0)
    T, C, taps = 7, 3, 4
    u, w, b = rng.standard_normal((T, C)), rng.standard_normal((C, taps)), rng.standard_normal(C)
    want = np.zeros((T, C))
    for t in range(T):
        for c in range(C):
            want[t, c] = b[c] + sum(w[c, taps - 1 - k] * u[t - k, c] for k in range(taps) if t - k >= 0)
    np.testing.assert_allclose(R.causal_conv(u, w, b), want, atol=1e-12)
    np.testing.assert_allclose(R.causal_conv(u, w[:, -1:], b), u * w[:, -1] + b)
    r, i, lam = R.sigmoid(rng.standard_normal((T, C))), R.sigmoid(rng.standard_normal((T, C))), rng.standard_normal(C)
    S, got = np.zeros(C), R.gated_linear_recurrence(u, r, i, lam)
    for t in range(T):
        for c in range(C):
            a = math.exp(-8.0 * r[t, c] * math.log(1 + math.exp(lam[c])))
            S[c] = a * S[c] + math.sqrt(1 - a * a) * i[t, c] * u[t, c]
        np.testing.assert_allclose(got[t], S, atol=1e-12)
    M = rng.standard_normal((2, 3, 3))
    x = rng.standard_normal((4, 6))
    np.testing.assert_allclose(R.block_diagonal(x, M, np.zeros((2, 3)))[1, 3:], M[1] @ x[1, 3:])


def test_forward_projects_the_embedding_in_once_a_pass():
    cfg = arch_synth.momedra_config(16, 12, [AT(2, 1, 4, 4, ff=8), RG(6, 2)], loop=(0, 1, 3))
    t = {k: v.astype(np.float64) for k, v in arch_synth.momedra_weights(cfg, seed=2).items()}
    toks = [3, 1, 4, 1, 5]
    taps = []
    R.forward(cfg, t, toks, taps=taps)
    assert len(taps) == 4
    x0, eps, m = t["embed"][toks], cfg["norm"]["eps"], cfg["residual_mult"]
    x = x0
    for k in range(3):
        x = R.layer(x @ t["loop.in"][:, :16].T + x0 @ t["loop.in"][:, 16:].T, cfg["layers"][0], t, 0, eps, m)
        np.testing.assert_allclose(taps[k], x)
    # both sublayers read the same norm's output
    h = R.layer_norm(x0, t["l0.norm1"], eps)
    np.testing.assert_allclose(R.layer(x0, cfg["layers"][0], t, 0, eps, m),
                               x0 + m * (R.attention(h, cfg["layers"][0]["mixer"], t, "l0.mix.", eps) + R.unit(h, t, "l0.mlp.")))
    # a later position never changes an earlier one
    np.testing.assert_allclose(R.forward(cfg, t, toks)[:3], R.forward(cfg, t, toks[:3]), atol=1e-10)
