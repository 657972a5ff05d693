"""The Muzasun design without a GPU: configuration reading and its error messages, the tensor declaration, cache needs, load-time
fusion, and the plain implementation against second forms of its own mechanisms."""
import copy
import dataclasses
import math

import numpy as np
import pytest
import torch

import herbert_rs_b200 as hb
import muzasun_util as U
import plain_muzasun as P
from herbert_rs_b200.cache import SequenceCache
from herbert_rs_b200.config.muzasun import MuzasunConfig
from herbert_rs_b200.config.specs import ScaledRotarySpec
from herbert_rs_b200.errors import ConfigError, WeightError
from herbert_rs_b200.weights.loader import build_model, check_tensors, fill_model
from herbert_rs_b200.weights.safetensors_io import ModelFiles

F64 = torch.float64


def test_configuration_is_read_from_the_nested_keys():
    cfg = U.config([(U.attention(heads=6, kv_heads=3, dim=24, vdim=40, rot_dims=10, base=777.0), U.dense(ff=56)),
                    (U.mlstm(heads=5, dim=12, vdim=28, cap=3.5), None),
                    (U.delta(heads=6, kv_heads=2, dim=20, vdim=8, conv=5), U.moe(experts=7, top=3, ff=24, shared=32)),
                    (U.attention(heads=3, kv_heads=3, dim=8, vdim=40, v_mix=True), U.moe(shared=0)),
                    (U.attention(v_mix=False), None)], vocab=99, width=72, eps=3e-6, mult=0.7, logit_scale=2.5)
    spec = MuzasunConfig.from_dict(cfg).model_spec()
    assert (spec.vocab_size, spec.hidden_size, spec.logit_scale, spec.architecture) == (99, 72, 2.5, "Muzasun")
    assert [s.layer for s in spec.schedule] == [0, 1, 2, 3, 4]
    b0, b1, b2, b3, b4 = spec.blocks
    assert (b0.kind, b0.residual_mult, b0.norm1.kind, b0.norm2.weight_name, spec.final_norm.kind) == ("parallel", 0.7, "dynamic_tanh", "norm2", "dynamic_tanh")
    assert b1.ffn is None and b1.norm2 is None
    a = b0.mixer
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.qk_norm.eps, a.qk_norm.dim) == (6, 3, 24, 40, 3e-6, 24)
    assert a.bias and a.output_bias and a.head_qk_norm and a.position == ScaledRotarySpec(10, 777.0) and a.scale == 1 / math.sqrt(24)
    assert [b.mixer.value_blend for b in (b0, b3, b4)] == ["keep", "blend", None]
    m = b1.mixer
    assert (m.num_heads, m.key_dim, m.value_dim, m.gate_cap, m.norm_eps) == (5, 12, 28, 3.5, 3e-6)
    d = b2.mixer
    assert (d.num_heads, d.qk_heads, d.key_dim, d.value_dim, d.conv_taps, d.norm_eps) == (6, 2, 20, 8, 5, 3e-6)
    r = b2.ffn
    assert (r.num_experts, r.top_k, r.expert_size, r.shared.intermediate_size, r.score, r.renormalize, r.weigh_input) == (7, 3, 24, 32, "sigmoid", False, True)
    assert b3.ffn.shared is None
    assert hb.registry.architecture_for(cfg) == "Muzasun"
    assert "l1.norm2.alpha" in spec.unused_names and "l4.mix.vmix" in spec.unused_names and "l0.mix.vmix" not in spec.unused_names
    del cfg["logit_scale"], cfg["residual_mult"], cfg["layers"][0]["mixer"]["rot"]
    spec = MuzasunConfig.from_dict(cfg).model_spec()
    assert spec.logit_scale == 1.0 and spec.blocks[0].residual_mult == 1.0 and spec.blocks[0].mixer.position is None


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=25), "v_mix"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "unknown feed-forward kind"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=9), "router.top"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(edit, message):
    cfg = U.config([(U.attention(), U.dense()), (U.mlstm(), None), (U.delta(), U.moe()), (U.attention(), None)])
    edit(cfg)
    with pytest.raises(ConfigError, match=message):
        MuzasunConfig.from_dict(cfg)


def test_declared_tensors_and_cache_need(tmp_path):
    cfg = U.config([(U.attention(heads=4, kv_heads=2, dim=12, vdim=20), U.dense()), (U.mlstm(heads=3, dim=10, vdim=15), None),
                    (U.delta(heads=4, kv_heads=2, dim=6, vdim=9, conv=4), U.moe()), (U.delta(conv=1), U.moe(shared=0)), (U.attention(v_mix=False), None)])
    model = build_model(cfg, hb.Runtime("cpu", torch.bfloat16))
    specs, t = model.param_specs(), U.weights(cfg)
    assert set(specs) == set(t)
    for k, ps in specs.items():
        assert len(ps.shape) == t[k].dim() and all(a in (-1, b) for a, b in zip(ps.shape, t[k].shape)), k
    assert specs["l0.norm1.alpha"].shape == () and "l1.norm2" not in specs and "l4.mix.vmix" not in specs
    needs = model.cache_needs()
    assert (needs[0].kv.num_kv_heads, needs[0].kv.head_dim, needs[0].kv.planes, needs[0].kv.window) == (2, 32, 2, None)
    # values, a column of ones, zeros up to a multiple of eight; the running maximum beside it
    assert tuple(needs[1].state.shape) == (3, 10, 16) and dict(needs[1].states)["running_max"].shape == (3,)
    assert tuple(needs[2].state.shape) == (4, 6, 9) and dict(needs[2].states)["conv"].shape == (3, 2 * 2 * 6 + 4 * 9)
    assert needs[3].states == () and needs[1].kv is None
    cache = SequenceCache(needs, model.reads_cache_of(), num_pages=8, num_slots=2, page_size=16)
    assert cache.step_kv[0] != cache.step_kv[4]
    U.write(cfg, t, tmp_path)
    assert P.PlainMuzasun(str(tmp_path)).logits([1, 2, 3]).shape == (3, 131)


def test_a_missing_misshapen_or_strange_tensor_is_reported_and_an_unused_one_is_not(tmp_path):
    cfg = U.config([(U.attention(), U.dense()), (U.mlstm(), None), (U.delta(), U.moe()), (U.attention(v_mix=False), None)])
    t = U.weights(cfg)
    t["l1.norm2"], t["l3.mix.vmix"] = torch.zeros(64), torch.zeros(())            # no use is made of these
    U.write(cfg, t, tmp_path / "fine")
    files = ModelFiles(str(tmp_path / "fine"))
    check_tensors(build_model(cfg, hb.Runtime("cpu", torch.bfloat16)), files)
    files.close()
    del t["l1.mix.f.b"], t["final.norm.alpha"]
    t["l0.norm2.alpha"] = t["l0.norm2.alpha"].reshape(1)
    t["l2.mix.k"] = t["l2.mix.k"][:-1].contiguous()
    t["l2.mix.extra"] = torch.zeros(3)
    U.write(cfg, t, tmp_path / "bad")
    files = ModelFiles(str(tmp_path / "bad"))
    with pytest.raises(WeightError) as e:
        check_tensors(build_model(cfg, hb.Runtime("cpu", torch.bfloat16)), files)
    files.close()
    assert all(n in str(e.value) for n in ("l1.mix.f.b", "final.norm.alpha", "l0.norm2.alpha", "l2.mix.k", "l2.mix.extra"))


def test_load_time_fusion_and_the_factor_on_the_logits():
    cfg = U.config([(U.delta(heads=3, kv_heads=1, dim=5, vdim=7, rank=6), None), (U.mlstm(heads=1, dim=3, vdim=2), None)], logit_scale=3.0)
    t = U.weights(cfg)
    for dtype, parts in ((torch.bfloat16, 2), (torch.float32, 1)):
        rt = hb.Runtime("cpu", dtype)
        model = build_model(cfg, rt)
        fill_model(model, lambda n: t[n], rt)
        d, m = model.blocks[0].mixer, model.blocks[1].mixer
        assert d.w_in.shape[0] % 8 == 0 and m.w_in.shape[0] % 8 == 0        # rows that start on 16 bytes
        low = torch.randn(4, 6 + 9)
        x = torch.cat([low[:, :6]] * parts + [low[:, 6:]], dim=1)
        if parts > 1:                                                       # the inner rows' two parts add up
            x[:, :6] *= 0.75
            x[:, 6:12] *= 0.25
            x = torch.cat([x, torch.zeros(4, d.w_low.shape[1] - x.shape[1])], dim=1)
            assert d.w_low.shape[1] % 8 == 0
        wide = x @ d.w_low.float().T
        want = torch.cat([low[:, :6] @ t["l0.mix.a2"].float().T, low[:, 6:] @ t["l0.mix.g2"].float().T], dim=1)
        assert (wide - want).abs().max() < 1e-5
        assert not model.scale_logits and (model.final_norm.bias - 3.0 * t["final.norm.b"].float()).abs().max() < 1e-6
        assert (model.final_norm.weight - 3.0 * t["final.norm"].float()).abs().max() < 1e-6
    t["l0.mix.a2"] = t["l0.mix.a2"][:, :-1].contiguous()
    with pytest.raises(WeightError, match="a1 has 6 rows but a2"):
        rt = hb.Runtime("cpu", torch.bfloat16)
        fill_model(build_model(cfg, rt), lambda n: t[n], rt)


def test_options_that_do_not_go_together_are_refused():
    rt = hb.Runtime("cpu", torch.bfloat16)
    from herbert_rs_b200.parts import AttentionMixer
    a = MuzasunConfig.from_dict(U.config([(U.attention(), None)])).layers[0][0]
    AttentionMixer(a, rt)
    for change in (dict(qk_norm=None), dict(whole_qk_norm=True), dict(difference=0.3), dict(value_blend="other"), dict(conv_taps=3), dict(sink=True)):
        with pytest.raises(ConfigError):
            AttentionMixer(dataclasses.replace(a, **change), rt)
    moe = MuzasunConfig.from_dict(U.config([(U.mlstm(), U.moe())])).layers[0][1]
    from herbert_rs_b200.parts import RoutedFeedForward
    with pytest.raises(ConfigError, match="gated experts only"):
        RoutedFeedForward(dataclasses.replace(moe, gated=False, expert_names=("e{e}.up", "e{e}.down")), rt)


def test_blocks_hand_norms_only_to_blocks_of_their_kind():
    """Two norms with statistics are no entry for the block before; one is, and norms without statistics are another kind."""
    from herbert_rs_b200.config.specs import NormSpec
    from herbert_rs_b200.parts import ParallelBlock
    rt = hb.Runtime("cpu", torch.bfloat16)
    b = MuzasunConfig.from_dict(U.config([(U.mlstm(), U.dense())])).model_spec().blocks[0]
    tanh = ParallelBlock(b, rt)
    assert tanh.chain_kind == "pointwise" and len(tanh.norms) == 2
    rms = NormSpec(64, 1e-5, weight_name="norm1")
    two = ParallelBlock(dataclasses.replace(b, norm1=rms, norm2=NormSpec(64, 1e-5, weight_name="norm2")), rt)
    assert two.chain_kind == "norm" and two.first_norm() is None
    one = ParallelBlock(dataclasses.replace(b, norm1=rms, norm2=None), rt)
    assert one.chain_kind == "norm" and one.first_norm() is one.norm1
    assert ParallelBlock(dataclasses.replace(b, ffn=None), rt).norms[1:] == []


# ---- the plain implementation against second forms of its mechanisms --------------------------------
def test_small_functions_against_torch():
    g = torch.Generator().manual_seed(0)
    F = torch.nn.functional
    x = torch.randn(5, 24, generator=g, dtype=F64) * 3
    w, b = 1 + 0.1 * torch.randn(24, generator=g, dtype=F64), torch.randn(24, generator=g, dtype=F64)
    assert (P.unit_rms(x, 1e-5) - F.rms_norm(x, (24,), None, 1e-5)).abs().max() < 1e-12
    assert (P.silu(x) - F.silu(x)).abs().max() < 1e-12 and (P.softplus(x * 30) - torch.logaddexp(x * 30, torch.zeros_like(x))).abs().max() < 1e-12
    assert (P.log_sigmoid(x * 20) - F.logsigmoid(x * 20)).abs().max() < 1e-12
    cw = torch.randn(24, 4, generator=g, dtype=F64)
    ref = F.conv1d(F.pad(x.T[None], (3, 0)), cw[:, None, :], groups=24)[0].T
    assert (P.causal_conv(x, cw) - ref).abs().max() < 1e-12 and (P.causal_conv(x[:2], cw) - ref[:2]).abs().max() < 1e-12
    y = P.squash_norm(x, torch.tensor(0.7, dtype=F64), w, b)
    assert abs(float(y[2, 3]) - (math.tanh(0.7 * float(x[2, 3])) * float(w[3]) + float(b[3]))) < 1e-14
    assert (P.unit_vector(x).norm(dim=-1) - 1).abs().max() < 1e-6 and P.capped(x * 100, 4.0).abs().max() <= 4.0


def test_rotation_makes_scores_depend_on_distance_only():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 2, 16, generator=g, dtype=F64), torch.randn(1, 2, 16, generator=g, dtype=F64)

    def score(i, j):
        return float((P.rotate(q, [i], 100.0, 8)[0, 0] * P.rotate(k, [j], 100.0, 8)[0, 0]).sum())
    assert abs(score(10, 3) - score(107, 100)) < 1e-9 and abs(score(10, 3) - score(10, 4)) > 1e-3
    r = P.rotate(q, [5], 100.0, 8)[0, 1]
    a = 5 * 100.0 ** (-2 / 8)
    assert torch.equal(r[8:], q[0, 1, 8:]) and abs(float(r[1]) - float(q[0, 1, 1] * math.cos(a) - q[0, 1, 5] * math.sin(a))) < 1e-12


def test_the_matrix_memory_against_sums_without_a_running_maximum_and_from_a_saved_state():
    """Unscaled: weights e^(i_s + f_(s+1) + .. + f_t), and a floor of 1 under |n . q| where the running maximum is folded out."""
    g = torch.Generator().manual_seed(3)
    T, H, d, e = 13, 2, 4, 3
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (d, d, e))
    i, f = 3 * torch.randn(T, H, generator=g, dtype=F64), P.log_sigmoid(2 * torch.randn(T, H, generator=g, dtype=F64))
    o, (S, n, m) = P.matrix_memory(q, k, v, i, f)
    run = torch.zeros(H, dtype=F64)
    for t in range(T):
        run = torch.maximum(run + f[t], i[t])
        for h in range(H):
            w = torch.tensor([math.exp(float(i[s, h] + f[s + 1:t + 1, h].sum())) for s in range(t + 1)], dtype=F64)
            sc = w * (k[:t + 1, h] @ q[t, h])
            top = (sc[:, None] * v[:t + 1, h]).sum(0)
            scale = math.exp(-float(run[h]))
            bottom = max(abs(float(sc.sum())), 1.0) + P.READ_EPS / scale
            assert (o[t, h] - top / bottom).abs().max() < 1e-10
    assert (m - run).abs().max() < 1e-12
    o1, s1 = P.matrix_memory(q[:5], k[:5], v[:5], i[:5], f[:5])
    o2, s2 = P.matrix_memory(q[5:], k[5:], v[5:], i[5:], f[5:], *s1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12 and (s2[0] - S).abs().max() < 1e-12


def test_the_channel_delta_rule_as_products_of_matrices():
    """S_t = (I - beta k k^T) diag(g) S + beta k v^T."""
    g = torch.Generator().manual_seed(4)
    T, H, d, e = 9, 2, 5, 3
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (d, d, e))
    dec, beta = torch.rand(T, H, d, generator=g, dtype=F64), torch.rand(T, H, generator=g, dtype=F64)
    o, S = P.channel_delta(q, k, v, dec, beta)
    for h in range(H):
        X = torch.zeros(d, e, dtype=F64)
        for t in range(T):
            kk = k[t, h]
            X = (torch.eye(d, dtype=F64) - beta[t, h] * torch.outer(kk, kk)) @ torch.diag(dec[t, h]) @ X + beta[t, h] * torch.outer(kk, v[t, h])
            assert (o[t, h] - X.T @ q[t, h]).abs().max() < 1e-12
        assert (X - S[h]).abs().max() < 1e-12
    o1, S1 = P.channel_delta(q[:4], k[:4], v[:4], dec[:4], beta[:4])
    o2, _ = P.channel_delta(q[4:], k[4:], v[4:], dec[4:], beta[4:], S1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12


def test_the_mixture_token_by_token():
    cfg = U.config([(U.mlstm(), U.moe(experts=5, top=2))])
    W = {k: v.double() for k, v in U.weights(cfg, 3).items()}
    h = torch.randn(7, 64, dtype=F64)
    f = cfg["layers"][0]["mlp"]
    y = P.mixture_ff(h, W, "l0.mlp.", f, F64, lambda t: t)
    for t in range(7):
        s = torch.sigmoid(W["l0.mlp.router"] @ h[t])
        best = sorted(range(5), key=lambda e: -float(s[e]))[:2]
        want = torch.zeros(64, dtype=F64)
        for p, x in [(f"l0.mlp.e{e}.", float(s[e]) * h[t]) for e in best] + [("l0.mlp.shared.", h[t])]:
            want += W[p + "down"] @ (torch.nn.functional.silu(W[p + "gate"] @ x) * (W[p + "up"] @ x))
        assert (y[t] - want).abs().max() < 1e-10


def test_leaving_out_a_mechanism_moves_the_logits():
    layers = [(U.attention(rot_dims=8, sharp=2.0), U.dense()), (U.mlstm(), U.moe()), (U.delta(), U.dense()), (U.attention(sharp=2.0), U.moe())]
    cfg = U.config(layers)
    pm = P.PlainMuzasun(config=cfg, tensors=U.weights(cfg, 8))
    ids = np.random.default_rng(5).integers(0, 131, 40).tolist()
    ref = pm.logits(ids)
    low = float((pm.logits(ids, F64, P.bf16_storage) - ref).abs().max())

    def moved(cfg=None, W=None):
        return float((P.PlainMuzasun(config=cfg or pm.cfg, tensors=W or pm.W).logits(ids) - ref).abs().max())

    def edited(fn):
        c = copy.deepcopy(pm.cfg)
        fn(c)
        return c
    first, mem, rule, second = (lambda c, i=i: c["layers"][i]["mixer"] for i in range(4))
    for what, fn in {
        "multiplier": lambda c: c.update(residual_mult=0.6), "logits": lambda c: c.update(logit_scale=1.6), "no rotation": lambda c: first(c).pop("rot"),
        "all rotated": lambda c: first(c)["rot"].update(dims=16), "base": lambda c: second(c)["rot"].update(base=50.0), "scale": lambda c: first(c).update(scale=0.2),
        "no blending": lambda c: second(c).update(v_mix=False), "cap": lambda c: mem(c).update(gate_cap=1.0), "top": lambda c: c["layers"][1]["mlp"]["router"].update(top=1),
        "no shared expert": lambda c: c["layers"][3]["mlp"].pop("shared"), "no feed-forward": lambda c: c["layers"][2].update(mlp=None),
    }.items():
        assert moved(edited(fn)) > 3 * low, what
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l3.mix.o.b", "l1.mix.f.b", "l2.mix.dt_bias", "l2.mix.A_log", "l2.mix.b", "l0.norm1.b", "l1.norm2.b", "final.norm.b"):
        assert moved(W=dict(pm.W, **{name: torch.zeros_like(pm.W[name])})) > 3 * low, name
    for name in ("l0.mix.q.norm", "l3.mix.k.norm", "l1.mix.norm", "l2.mix.norm", "l2.mix.k.conv", "l3.mix.vmix", "l0.norm1.alpha", "l2.norm2.alpha", "final.norm.alpha"):
        assert moved(W=dict(pm.W, **{name: pm.W[name] * 0.6})) > 3 * low, name
    assert moved(W=dict(pm.W, **{"l0.mix.vmix": pm.W["l0.mix.vmix"] * 0.0})) == 0.0       # the first such layer makes no use of its own
    swapped = dict(pm.W, **{"l0.norm1": pm.W["l0.norm2"], "l0.norm2": pm.W["l0.norm1"]})
    assert moved(W=swapped) > 3 * low                                                     # each sublayer has its own norm
