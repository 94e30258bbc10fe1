"""Host-side pieces of the Sozanex family (no GPU): configuration reading, the order of layer runs, scaled rotary frequencies,
weight regrouping, cache sizing, the registry, and checks of the float64 oracle against second formulations."""
import math
import warnings

import pytest
import torch

import sozanex_oracle as O
from torchao_fork_b200._models import registry
from torchao_fork_b200._models.rotary import BandScaling, RotaryArgs, RotaryScaling
from torchao_fork_b200._models.sozanex import Sozanex, SozanexArgs, sozanex_configs
from torchao_fork_b200._models.sozanex.model import NO_WINDOW

F64 = torch.float64


def _cfg(loop=(1, 3, 2)):
    return O.model_config([O.latent_layer(ramp=(4.0, 64, 8.0, 1.0)), O.attention_layer(bands=(4.0, 64, 1.0, 4.0)), O.latent_layer(ff=0),
                           O.attention_layer(size=5)], loop=loop)


def test_configuration_round_trip_and_absent_parts():
    cfg = _cfg()
    a = SozanexArgs.from_dict(cfg)
    assert a.to_dict() == cfg and SozanexArgs.from_dict(a.to_dict()) == a
    assert isinstance(a.layers[0].mixer.rot.scaling, RotaryScaling) and isinstance(a.layers[1].mixer.rot.scaling, BandScaling)
    assert a.layers[2].ff == 0 and a.bigram.mul_cur == 11 and a.layers[0].mixer.window == NO_WINDOW and a.layers[3].mixer.window == 5
    bare = O.model_config([O.attention_layer(rot=0, size=0)])
    del bare["embedding"]
    b = SozanexArgs.from_dict(bare)
    assert b.layers[0].mixer.window == NO_WINDOW and b.layers[0].mixer.rot.dims == 0
    assert b.embedding_scale == 1.0 and b.bigram is None and b.loop is None
    for name, make in sozanex_configs.items():
        assert SozanexArgs.from_dict(make().to_dict()) == make(), name


def test_bad_configurations_are_refused():
    for layer, key, value in ((1, "kv_heads", 3), (0, "kv_rank", 513), (1, "vdim", 257)):
        cfg = _cfg()
        cfg["layers"][layer]["mixer"][key] = value
        with pytest.raises(AssertionError):
            SozanexArgs.from_dict(cfg)
    for loop in ((2, 2, 1), (0, 5, 1), (1, 2, 0)):
        with pytest.raises(AssertionError):
            SozanexArgs.from_dict(_cfg(loop))
    for edit in (lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][0]["mlp"].update(kind="moe")):
        cfg = _cfg()
        edit(cfg)
        with pytest.raises(NotImplementedError):
            SozanexArgs.from_dict(cfg)


@pytest.mark.parametrize("loop,runs", [(None, [0, 1, 2, 3]), ((0, 4, 1), [0, 1, 2, 3]), ((1, 3, 2), [0, 1, 2, 1, 2, 3]),
                                       ((0, 1, 3), [0, 0, 0, 1, 2, 3]), ((3, 4, 2), [0, 1, 2, 3, 3])])
def test_order_of_layer_runs_and_beginnings_of_passes(loop, runs):
    a = SozanexArgs.from_dict(_cfg(loop))
    assert a.runs == runs and a.schedule == O.order(_cfg(loop))
    assert sum(begins for _, begins in a.schedule) == (loop[2] if loop else 0)


@pytest.mark.parametrize("dims,base,bands", [(24, 7e3, (5.0, 600, 1.0, 3.5)), (8, 500.0, (8.0, 64, 0.5, 9.0)), (6, 30.0, (2.0, 20, 1.0, 1.5)), (2, 9.0, (3.0, 7, 2.0, 5.0))])
def test_band_scaled_frequencies(dims, base, bands):
    r = O.rotary(dims, base, bands=bands)
    f, amp = O.frequencies(r)
    got = RotaryArgs.from_dict(r)
    assert torch.allclose(got.inv_freq("cpu"), f.float(), rtol=1e-6) and amp == 1.0 == got.amplitude
    plain = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    wave = 2 * math.pi / plain
    factor, original, low, high = bands
    assert torch.equal(f[wave < original / high], plain[wave < original / high])
    slow = wave > original / low
    assert torch.allclose(f[slow], plain[slow] / factor, rtol=1e-12)
    mid = ~slow & (wave >= original / high)
    s = (original / wave[mid] - low) / (high - low)
    assert torch.allclose(f[mid], (1 - s) * plain[mid] / factor + s * plain[mid], rtol=1e-12)


@pytest.mark.parametrize("dims,base,ramp", [(14, 3e4, (3.0, 900, 24.0, 1.5)), (4, 1e6, (2.0, 16, 4.0, 3.9)), (6, 50.0, (8.0, 40, 2.0, 0.5))])
def test_ramp_scaled_frequencies(dims, base, ramp):
    r = O.rotary(dims, base, ramp=ramp)
    f, amp = O.frequencies(r)
    got = RotaryArgs.from_dict(r)
    assert torch.allclose(got.inv_freq("cpu"), f.float(), rtol=1e-6) and abs(got.amplitude - amp) < 1e-12
    assert abs(amp - (1 + 0.1 * math.log(ramp[0]))) < 1e-12


def test_weights_are_regrouped_and_checked_against_the_configuration():
    cfg = _cfg()
    w = O.random_weights(cfg, 0)
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        m = Sozanex(SozanexArgs.from_dict(cfg), w, "cpu", torch.float32)
    lat, att, W = m.layers[0], m.layers[1], 32
    assert torch.equal(m.loop_in[:W], w["loop.in"][:, :W].float()) and torch.equal(m.loop_in[W:], w["loop.in"][:, W:].float())
    assert lat.w_in.shape == (3 * 12 + 10 + 14 + 4, W) and torch.equal(lat.w_in[lat.kv_off:], w["l0.mix.dkv"].float())
    assert torch.equal(lat.w_in[lat.g_off:lat.g_off + 36], w["l0.mix.g"].float()) and lat.uk.shape == (3, 8, 14) and lat.uv.shape == (3, 12, 14)
    assert att.w_in.shape == (4 * 12 + 2 * 12 + 2 * 8, W) and torch.equal(att.w_in[att.v_off:], w["l1.mix.v"].float())
    assert m.bigram.shape == (38, W) and not hasattr(m.layers[2], "w_up")
    with pytest.warns(UserWarning):
        Sozanex(SozanexArgs.from_dict(cfg), dict(w, extra=torch.zeros(1)), "cpu", torch.float32)
    bad = dict(w)
    bad["l0.mix.sink"] = torch.zeros(5)
    with pytest.raises(ValueError):
        Sozanex(SozanexArgs.from_dict(cfg), bad, "cpu", torch.float32)
    del bad["l0.mix.sink"]
    with pytest.raises(KeyError):
        Sozanex(SozanexArgs.from_dict(cfg), bad, "cpu", torch.float32)


def test_state_per_layer_run_growth_and_bounds():
    cfg = _cfg()
    m = Sozanex(SozanexArgs.from_dict(cfg), O.random_weights(cfg, 0), "cpu", torch.float32)
    m.setup_caches(2, 40)
    assert len(m.run_state) == 7                          # six layer runs and the embedding's last token
    assert m.run_state[0].latent.c.shape == (2, 40, 14) and m.run_state[1].window.k.shape == (2, 9, 24) and m.run_state[5].window.ring == 5
    assert m.run_state[1].window is not m.run_state[3].window and m.run_state[2].latent is not m.run_state[4].latent
    assert m.run_state[6].last.token.dtype == torch.int64 and m.states.max_seq_length == 40
    s = m.states.slot_of("a")
    m.states.extend(s, 40)
    with pytest.raises(RuntimeError):
        m.states.extend(s, 1)
    m.run_state[6].last.token[s] = 33
    m.states.slot_of("b"), m.states.slot_of("c")          # a third request doubles the slots of every state
    assert m.run_state[4].latent.kr.shape[0] == 4 and m.run_state[6].last.token.tolist() == [33, 0, 0, 0] and m.max_batch_size == 4
    only = O.model_config([O.attention_layer(size=6)], bigram=None)
    m = Sozanex(SozanexArgs.from_dict(only), O.random_weights(only, 0), "cpu", torch.float32)
    m.setup_caches(1, 8)
    assert len(m.run_state) == 1 and m.states.max_seq_length == 1 << 30      # nothing was cut: a sequence may go on


def test_registry_and_product_random_weights():
    fams = registry.families()
    assert "sozanex" in fams and "Sozanex-test" in fams["sozanex"].names()
    cfg = sozanex_configs["Sozanex-test"]()
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        Sozanex(cfg, Sozanex.random_weights(cfg, "cpu", torch.float32), "cpu", torch.float32)     # a missing or unused tensor raises


# ------------------------------------------------------------------------------------------------ the oracle against itself
def test_oracle_sink_takes_its_share_of_uniform_weights():
    T = 5
    z, v = torch.zeros(T, 1, 2, dtype=F64), torch.ones(T, 1, 1, dtype=F64)
    out = O.sink_softmax(z, z, v, 1.0, sink=torch.tensor([math.log(3.0)], dtype=F64))
    for i in range(T):
        assert float(out[i, 0, 0]) == pytest.approx((i + 1) / (i + 4))
    win = O.sink_softmax(z, z, torch.arange(T, dtype=F64).view(T, 1, 1), 1.0, size=2)
    assert win.view(-1).tolist() == [0.0, 0.5, 1.5, 2.5, 3.5]


def test_oracle_embedding_reads_the_pair_and_the_first_row():
    cfg = O.model_config([], width=4, vocab=9, scale=2.0, bigram=(7, 3, 5))
    w = {k: v.double() for k, v in O.random_weights(cfg, 1).items()}
    x = O.embedding(cfg, w, [4, 8, 8])
    assert torch.equal(x[0], 2 * w["embed"][4] + w["bigram"][7])
    assert torch.equal(x[1], 2 * w["embed"][8] + w["bigram"][(4 * 3 + 8 * 5) % 7])
    assert torch.equal(x[2], 2 * w["embed"][8] + w["bigram"][(8 * 3 + 8 * 5) % 7])


def test_oracle_rotation_depends_on_distance_only_and_keeps_the_rest():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 10, generator=g, dtype=F64), torch.randn(1, 1, 10, generator=g, dtype=F64)
    for layout, rot in (("half", O.rotary(8, 90.0, bands=(4.0, 64, 1.0, 4.0))), ("interleaved", O.rotary(6, 90.0))):
        at = lambda x, p: O.rotate(x, torch.tensor([p]), rot, layout)
        assert torch.allclose((at(q, 9) * at(k, 4)).sum(), (at(q, 105) * at(k, 100)).sum())
        assert torch.equal(at(q, 9)[..., rot["dims"]:], q[..., rot["dims"]:])


def test_oracle_layer_norm_and_squared_relu():
    x = torch.tensor([[1.0, 2.0, 6.0]], dtype=F64)
    assert torch.allclose(O.layer_norm(x, torch.ones(3, dtype=F64), 0.0), (x - 3) / math.sqrt(14 / 3))
    assert O.squared_relu(torch.tensor([-2.0, 0.0, 3.0])).tolist() == [0.0, 0.0, 9.0]
