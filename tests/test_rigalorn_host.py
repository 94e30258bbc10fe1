"""Host-side pieces of the Rigalorn family (no GPU): configuration reading, scaled rotary frequencies, weight regrouping,
cache sizing, the step's tables for latent attention, the registry, and checks of the float64 oracle against a second
formulation of the same mechanism."""
import math
import warnings

import numpy as np
import pytest
import torch

import rigalorn_oracle as O
from torchao_fork_b200._models import registry
from torchao_fork_b200._models.rigalorn import Rigalorn, RigalornArgs, rigalorn_configs
from torchao_fork_b200._models.rigalorn.model import NO_WINDOW
from torchao_fork_b200._models.rigalorn.step import StepEngine
from torchao_fork_b200._models.rotary import RotaryArgs

F64 = torch.float64


def _cfg():
    return O.model_config([O.attention_layer(v_mix=True, scaling=(4.0, 64, 8.0, 1.0)), O.delta_layer(), O.latent_layer(ff=0),
                           O.attention_layer(v_mix=True, size=5)])


def test_configuration_round_trip_and_absent_parts():
    cfg = _cfg()
    a = RigalornArgs.from_dict(cfg)
    assert a.to_dict() == cfg and RigalornArgs.from_dict(a.to_dict()) == a
    assert a.first_v_mix == 0 and a.layers[2].ff == 0 and a.layers[0].mixer.rot.scaling.original == 64
    bare = O.model_config([O.attention_layer(rot=0, size=0), O.latent_layer(size=0)])
    del bare["embedding"]
    b = RigalornArgs.from_dict(bare)
    assert b.layers[0].mixer.window == NO_WINDOW == b.layers[1].mixer.window and b.layers[0].mixer.rot.dims == 0
    assert b.embedding_scale == 1.0 and b.first_v_mix is None
    for name, make in rigalorn_configs.items():
        assert RigalornArgs.from_dict(make().to_dict()) == make(), name


def test_bad_configurations_are_refused():
    for layer, key, value in ((0, "kv_heads", 3), (1, "kv_heads", 3), (3, "vdim", 16), (2, "kv_rank", 513), (0, "vdim", 257)):
        cfg = _cfg()
        cfg["layers"][layer]["mixer"][key] = value
        with pytest.raises(AssertionError):
            RigalornArgs.from_dict(cfg)
    cfg = _cfg()
    cfg["layers"][0]["type"] = "unknown"
    with pytest.raises(NotImplementedError):
        RigalornArgs.from_dict(cfg)
    cfg = _cfg()
    cfg["layers"][0]["mlp"]["kind"] = "moe"
    with pytest.raises(NotImplementedError):
        RigalornArgs.from_dict(cfg)


@pytest.mark.parametrize("dims,base,scaling", [(8, 500.0, None), (64, 1e4, (4.0, 512, 32.0, 1.0)), (6, 50.0, (8.0, 40, 2.0, 0.5)),
                                               (4, 1e6, (2.0, 16, 4.0, 3.9)), (2, 300.0, (16.0, 4096, 32.0, 1.0))])
def test_scaled_rotary_frequencies_against_the_oracle(dims, base, scaling):
    r = O.rotary(dims, base, scaling)
    f, amp = O.frequencies(r)
    got = RotaryArgs.from_dict(r)
    assert torch.equal(got.inv_freq("cpu"), f.float()) and abs(got.amplitude - amp) < 1e-12
    plain = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    if scaling is None:
        assert amp == 1.0 and torch.allclose(f, plain)
    else:       # fast pairs at most keep their frequency, slow ones are at most `factor` times slower
        assert bool((f <= plain * (1 + 1e-12)).all()) and bool((f >= plain / scaling[0] * (1 - 1e-12)).all())
        assert abs(amp - (1 + 0.1 * math.log(scaling[0]))) < 1e-12


def test_weights_are_regrouped_and_checked_against_the_configuration():
    cfg = _cfg()
    w = O.random_weights(cfg, 0)
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        m = Rigalorn(RigalornArgs.from_dict(cfg), w, "cpu", torch.float32)
    a, d, l = m.layers[0], m.layers[1], m.layers[2]
    assert a.w_in.shape == (4 * 12 + 2 * 12 + 2 * 8 + 40, 32) and a.w_out.shape == (32, 4 * 8 + 40) and a.up_off == 88
    assert torch.equal(a.w_in[a.up_off:], w["l0.mlp.up"].float()) and torch.equal(a.w_out[:, 32:], w["l0.mlp.down"].float())
    assert d.w_in.shape == (2 * 2 * 8 + 4 * 12 + 4 * 12 + 40 + 4 + 4, 32) and d.conv_w.shape == (3, 2 * 2 * 8 + 4 * 12)
    assert torch.equal(d.w_in[d.b_off:], w["l1.mix.b"].float()) and torch.equal(d.w_in[d.a_off:d.b_off], w["l1.mix.a"].float())
    assert torch.equal(d.conv_w[:, 16:32].t(), w["l1.mix.k.conv"].float())
    assert l.w_in.shape == (10 + 14 + 4, 32) and l.w_out.shape == (32, 36) and l.uk.shape == (3, 8, 14) and l.uv.shape == (3, 12, 14)
    p, q = w["l0.mlp.act"].double().tolist()
    assert abs(a.act_pos - math.log1p(math.exp(p))) < 1e-12 and abs(a.act_neg - 0.5 - math.log1p(math.exp(q))) < 1e-12
    assert abs(m.layers[3].lam - float(w["l3.mix.vmix"])) < 1e-12
    with pytest.warns(UserWarning):
        Rigalorn(RigalornArgs.from_dict(cfg), dict(w, extra=torch.zeros(1)), "cpu", torch.float32)
    bad = dict(w)
    bad["l1.mix.A_log"] = torch.zeros(5)
    with pytest.raises(ValueError):
        Rigalorn(RigalornArgs.from_dict(cfg), bad, "cpu", torch.float32)
    del bad["l1.mix.A_log"]
    with pytest.raises(KeyError):
        Rigalorn(RigalornArgs.from_dict(cfg), bad, "cpu", torch.float32)


def test_state_sizes_growth_and_the_bound_of_a_cut_window():
    cfg = _cfg()
    w = O.random_weights(cfg, 0)
    m = Rigalorn(RigalornArgs.from_dict(cfg), w, "cpu", torch.float32)
    m.setup_caches(3, 100)
    assert m.run_state[0].window.k.shape == (3, 9, 2 * 12) and m.run_state[2].latent.c.shape == (3, 11, 14)
    assert m.run_state[1].mat.s.shape == (3, 4, 12, 8) and m.run_state[1].conv.x.shape == (3, 2, 80)
    assert m.states.max_seq_length == 1 << 30            # no window was cut: a sequence may go on
    m = Rigalorn(RigalornArgs.from_dict(cfg), w, "cpu", torch.float32)
    m.setup_caches(1, 10)
    assert m.run_state[2].latent.c.shape[1] == 10 and m.run_state[0].window.ring == 9 and m.states.max_seq_length == 10
    s = m.states.slot_of("a")
    m.states.extend(s, 10)
    with pytest.raises(RuntimeError):
        m.states.extend(s, 1)
    m.states.slot_of("b")                                # a second request doubles the slots of every state
    assert m.run_state[2].latent.kr.shape[0] == 2 and m.run_state[1].conv.x.shape[0] == 2 and m.max_batch_size == 2


def test_tables_of_the_expanded_latent_attention_name_every_visible_row_once():
    """Two sequences under a window of 5: one continues at position 7 in slot 2, one starts fresh in slot 0."""
    shape, form = ("latent", 2, 16, 16, 16, 16, 5), (64, 1 << 30, True)
    starts, counts = np.array([0, 70]), np.array([70, 3])
    slot, pos = np.array([2] * 70 + [0] * 3), np.concatenate([np.arange(7, 77), np.arange(3)])
    tiles = {form: (np.array([0, 64, 70], np.int32), np.array([64, 6, 3], np.int32))}
    out = StepEngine._piece_tables(StepEngine.__new__(StepEngine), starts, counts, slot, pos, {shape: form}, tiles)
    rows, key0 = out[("rows", 5)], out[("key0", 5)]
    assert rows[:4].tolist() == [-1 - (2 * 5 + p % 5) for p in (3, 4, 5, 6)] and rows[4:74].tolist() == list(range(70))
    assert rows[74:].tolist() == [70, 71, 72]
    assert key0.tolist() == [-3, -3, 74]                 # row of key p = key0 + p: key 3 in row 0; the fresh sequence from row 74
    fresh = StepEngine._piece_tables(StepEngine.__new__(StepEngine), starts[:1], counts[:1], slot[:70] * 0, pos[:70] - 7, {shape: form},
                                     {form: (np.array([0, 64], np.int32), np.array([64, 6], np.int32))})
    assert ("rows", 5) not in fresh and fresh[("key0", 5)].tolist() == [0, 0]      # the step's own rows are all there is


def test_registry_and_product_random_weights():
    fams = registry.families()
    assert "rigalorn" in fams and "Rigalorn-test" in fams["rigalorn"].names()
    cfg = rigalorn_configs["Rigalorn-test"]()
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        Rigalorn(cfg, Rigalorn.random_weights(cfg, "cpu", torch.float32), "cpu", torch.float32)     # a missing or unused tensor raises


# ------------------------------------------------------------------------------------------------ the oracle against itself
def test_oracle_delta_rule_equals_a_product_of_transition_matrices():
    """S_t = (I - beta k k^T) g S_(t-1) + beta k v^T, multiplied out from zero for the last token."""
    gen = torch.Generator().manual_seed(0)
    T, d, dv = 9, 4, 3
    q, k = torch.randn(T, 1, d, generator=gen, dtype=F64), O.unit_vector(torch.randn(T, 1, d, generator=gen, dtype=F64))
    v, g, beta = torch.randn(T, 1, dv, generator=gen, dtype=F64), torch.rand(T, 1, generator=gen, dtype=F64), torch.rand(T, 1, generator=gen, dtype=F64)
    got = O.delta_recurrence(q, k, v, g, beta)
    S = torch.zeros(d, dv, dtype=F64)
    for j in range(T):
        term = beta[j, 0] * torch.outer(k[j, 0], v[j, 0])
        for t in range(j + 1, T):
            term = g[t, 0] * (torch.eye(d, dtype=F64) - beta[t, 0] * torch.outer(k[t, 0], k[t, 0])) @ term
        S = S + term
    assert torch.allclose(got[-1, 0], S.T @ q[-1, 0], atol=1e-12)


def test_oracle_delta_rule_replaces_what_a_key_held():
    """Writing twice under one unit key with step 1 leaves the second value only."""
    k = torch.zeros(3, 1, 2, dtype=F64)
    k[:, 0, 0] = 1.0
    v = torch.tensor([[[1.0, 2.0]], [[3.0, 4.0]], [[5.0, 6.0]]], dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    assert torch.allclose(O.delta_recurrence(k, k, v, one, one), v)


def test_oracle_window_counts_and_xielu_is_smooth_at_zero():
    T, size = 30, 4
    z, v = torch.zeros(T, 1, 2, dtype=F64), torch.randn(T, 1, 3, dtype=F64, generator=torch.Generator().manual_seed(1))
    out = O.window_softmax(z, z, v, 1.0, size)           # uniform scores: the mean of the visible values
    for i in (0, 3, 4, 29):
        assert torch.allclose(out[i, 0], v[max(0, i - size + 1):i + 1, 0].mean(0))
    p, q = torch.tensor(0.3, dtype=F64), torch.tensor(-0.7, dtype=F64)
    x = torch.tensor([-1e-4, 0.0, 1e-4], dtype=F64)
    y = O.xielu(x, p, q)
    assert float(y[1]) == 0.0 and abs(float((y[2] - y[0]) / 2e-4) - 0.5) < 1e-4
    assert float(O.xielu(torch.tensor(-40.0, dtype=F64), p, q)) == pytest.approx((0.5 + math.log1p(math.exp(-0.7))) * 39.0 - 20.0)


def test_oracle_convolution_last_tap_meets_the_current_row():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    assert O.causal_conv(x, torch.tensor([[2.0, 3.0]], dtype=F64)).view(-1).tolist() == [3.0, 32.0, 320.0]
