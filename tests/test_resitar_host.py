"""Host-side checks for the Resitar family: the registry reads a model directory's config.json into the C structs (and the Python mirror fills the
same bytes), and the plain restatement the GPU tests lean on is itself checked mechanism by mechanism on hand-made cases (no GPU)."""
import ctypes as C
import json
import math
from importlib import import_module

import pytest
import torch

from oracle import resitar_oracle as O

D = torch.float64


def small_cfg():
    par = {"left": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 10, "scale": 0.3, "mask": {"size": 7}, "rot": {"base": 5000.0, "dims": 6}},
           "right": {"heads": 4, "vdim": 5, "state": 3, "groups": 2, "conv": 3, "norm_groups": 5}, "left_scale": 0.7, "right_scale": 1.1}
    par2 = {"left": {"heads": 4, "kv_heads": 1, "dim": 8, "vdim": 3, "scale": 0.25,
                     "rot": {"base": 900.0, "dims": 8, "scaling": {"factor": 5.0, "original": 40, "fast": 3.0, "slow": 0.5}}},
            "right": {"heads": 2, "dim": 9}, "left_scale": 1.2, "right_scale": 0.4}
    dense = {"kind": "dense", "ff": 17}
    moe = {"kind": "moe", "expert": {"ff": 7}, "router": {"experts": 5, "top": 2}}
    return {"architecture": "Resitar", "vocab": 31, "width": 12, "streams": 3, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "parallel", "mixer": par, "mlp": moe}, {"type": "parallel_2", "mixer": par2, "mlp": dense},
                       {"type": "parallel", "mixer": par, "mlp": None}, {"type": "parallel_2", "mixer": par2, "mlp": moe}]}


def read(lib, capi, cfg, path, room=8):
    (path / "config.json").write_text(json.dumps(cfg))
    c, specs = capi.b2_config(), (capi.b2_layer_spec * 8)()
    return lib.b2_config_from_dir(str(path).encode(), C.byref(c), specs, room), c, specs


def test_registry_reads_the_layer_list(pkg, lib, tmp_path):
    capi = import_module("aws-k8s-ansible-provisioner_b200.capi")
    eng = import_module("aws-k8s-ansible-provisioner_b200.engine")
    cfg = small_cfg()
    rc, c, specs = read(lib, capi, cfg, tmp_path)
    assert rc == 0, lib.b2_last_error()
    assert (c.arch, c.num_layers, c.hidden, c.vocab, c.tie_embeddings, c.streams) == (capi.ARCH_RESITAR, 4, 12, 31, 1, 3)
    assert (c.loop_start, c.loop_stop, c.loop_times) == (1, 3, 2) and abs(c.rms_eps - 1e-5) < 1e-11
    a, b = specs[0], specs[1]
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.rot_dims, a.rot_halves, a.rot_orig) == (capi.MIXER_CHUNK_AND_SSM, 6, 3, 10, 10, 7, 6, 1, 0)
    assert (a.s_heads, a.s_vdim, a.s_dim, a.s_groups, a.conv_taps, a.s_norm_groups) == (4, 5, 3, 2, 3, 5)
    assert abs(a.mix_left - 0.7) < 1e-6 and abs(a.mix_right - 1.1) < 1e-6 and abs(a.scale - 0.3) < 1e-6
    assert (a.ff, a.ff_dim, a.experts, a.top) == (capi.FF_TOP_SOFTMAX_EXPERTS, 7, 5, 2)
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.chunk, b.rot_dims, b.rot_halves, b.rot_orig) == (capi.MIXER_FULL_AND_TIMEMIX, 4, 1, 8, 3, 0, 8, 0, 40)
    assert (b.s_heads, b.s_dim, b.s_vdim, b.ff, b.ff_dim) == (2, 9, 9, capi.FF_SWIGLU, 17) and (b.rot_factor, b.rot_fast, b.rot_slow) == (5.0, 3.0, 0.5)
    assert specs[2].ff == capi.FF_NONE
    # the Python mirror fills the same bytes from the same dict, and reads them back into an equal layer list
    mine, again = (capi.b2_layer_spec * 4)(), (capi.b2_layer_spec * 4)()
    for sp, layer in zip(mine, cfg["layers"]):
        eng._fill_layer_spec(sp, dict(layer, _family="resitar"))
    assert bytes(mine) == bytes(specs)[:C.sizeof(mine)]
    for sp, layer in zip(again, [eng._layer_dict(specs[i], "resitar") for i in range(4)]):
        eng._fill_layer_spec(sp, dict(layer, _family="resitar"))
    assert bytes(again) == bytes(mine)
    ec = eng.EngineConfig.resitar(cfg)
    assert (ec.arch, ec.streams, ec.loop, ec.tie_embeddings) == ("resitar", 3, (1, 3, 2), True)


def test_registry_optional_keys_and_refusals(pkg, lib, tmp_path):
    capi = import_module("aws-k8s-ansible-provisioner_b200.capi")
    cfg = small_cfg()
    del cfg["loop"]
    m0, m1 = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    for k in ("kv_heads", "vdim", "mask", "rot"):
        del m0["left"][k]
    del m0["right"]["groups"], m0["right"]["norm_groups"], m0["left_scale"], m1["left"]["rot"]["scaling"]
    rc, c, specs = read(lib, capi, cfg, tmp_path)
    assert rc == 0, lib.b2_last_error()
    assert c.loop_times == 0
    assert (specs[0].kv_heads, specs[0].vdim, specs[0].chunk, specs[0].rot_dims, specs[0].s_groups, specs[0].s_norm_groups, specs[0].mix_left) == (6, 10, 0, 0, 1, 1, 1.0)
    assert (specs[1].rot_orig, specs[1].rot_factor) == (0, 1.0)
    for spoil, word in ((lambda k: k["layers"][0].update(type="parallel_3"), b"parallel_3"), (lambda k: k.pop("streams"), b"streams"),
                        (lambda k: k["layers"][0]["mixer"].pop("right"), b"right"), (lambda k: k["layers"][0]["mixer"]["right"].pop("state"), b"state"),
                        (lambda k: k["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("slow"), b"slow"), (lambda k: k["loop"].update(stop=9), b"loop"),
                        (lambda k: k["layers"][0]["mlp"].update(kind="glu"), b"glu"), (lambda k: k["layers"][0]["mlp"].pop("router"), b"router")):
        bad = small_cfg()
        spoil(bad)
        assert read(lib, capi, bad, tmp_path)[0] != 0 and word in lib.b2_last_error(), word
    assert read(lib, capi, small_cfg(), tmp_path, room=3)[0] != 0


def test_streams_by_hand():
    xs = torch.tensor([[1.0, 2.0], [10.0, 20.0]], dtype=D)
    assert O.streams_in(xs, torch.tensor([2.0, -1.0], dtype=D)).tolist() == [-8.0, -16.0]
    mix = torch.tensor([[1.0, 3.0], [0.0, 2.0]], dtype=D)       # from stream 0: all to 0, three times to 1; from stream 1: twice to 1
    got = O.streams_out(xs, mix, torch.tensor([5.0, 7.0], dtype=D), torch.tensor([1.0, -1.0], dtype=D))
    assert got.tolist() == [[1 + 5, 2 - 5], [3 + 20 + 7, 6 + 40 - 7]]


def test_rotations_and_scaled_frequencies_by_hand():
    x = torch.tensor([[1.0, 2.0, 3.0, 4.0, 5.0]], dtype=D)
    rot = {"base": 100.0, "dims": 4}
    c, s, c2, s2 = math.cos(3.0), math.sin(3.0), math.cos(0.3), math.sin(0.3)
    assert torch.allclose(O.rotate(x, 3, rot, True), torch.tensor([[c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 5.0]], dtype=D))
    assert torch.allclose(O.rotate(x, 3, rot, False), torch.tensor([[c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5.0]], dtype=D))
    # pairs 0 .. 7 of base 2^16, 16 dims: f_i = 4^-i; over 1024 positions pair i turns 163 * 4^-i times
    sc = {"factor": 4.0, "original": 1024, "fast": 20.0, "slow": 2.0}
    f, mul = O.frequencies({"base": 65536.0, "dims": 16, "scaling": sc})
    lo, hi = math.floor(math.log(1024 / (2 * math.pi * 20)) / math.log(4)), math.ceil(math.log(1024 / (2 * math.pi * 2)) / math.log(4))
    assert (lo, hi) == (1, 4) and abs(mul - (1 + 0.1 * math.log(4))) < 1e-12
    for i in range(8):
        r = min(max((i - 1) / 3, 0), 1)
        assert abs(f[i] - 4.0 ** -i * (r / 4 + 1 - r)) < 1e-15
    # an empty ramp is a step
    f, _ = O.frequencies({"base": 65536.0, "dims": 16, "scaling": dict(sc, fast=1e9, slow=1e9)})
    assert f[0] == 1.0 and abs(f[1] - 1 / 16) < 1e-15


def test_attention_sees_its_chunk_only():
    keys, values = torch.eye(3, dtype=D), torch.tensor([[1.0], [2.0], [4.0]], dtype=D)
    q = torch.tensor([1.0, 2.0, 0.0], dtype=D)
    p = torch.softmax(torch.tensor([0.5, 1.0, 0.0], dtype=D), 0)
    assert torch.allclose(O.attention_step(q, keys, values, 0, 0.5), (p @ values))
    assert torch.allclose(O.attention_step(q, keys, values, 2, 0.5), values[2])


def test_recurrences_by_hand():
    S = torch.tensor([[1.0, 2.0], [0.0, -1.0]], dtype=D)
    x, B, Cv = torch.tensor([3.0, -2.0], dtype=D), torch.tensor([0.5, 1.0], dtype=D), torch.tensor([1.0, 2.0], dtype=D)
    d, a_log, Dk = torch.tensor(0.4, dtype=D), torch.tensor(math.log(2.0), dtype=D), torch.tensor(10.0, dtype=D)
    S1, y = O.ssm_step(S, x, B, Cv, d, a_log, Dk)
    want = math.exp(-0.8) * S + 0.4 * torch.outer(B, x)
    assert torch.allclose(S1, want) and torch.allclose(y, want[0] + 2 * want[1] + 10 * x)       # the read-out sees the write
    r, k, v = torch.tensor([1.0, 1.0], dtype=D), torch.tensor([0.6, 0.8], dtype=D), torch.tensor([3.0, -2.0], dtype=D)
    w, u = torch.tensor([0.5, 0.25], dtype=D), torch.tensor([2.0, 0.0], dtype=D)
    S2, o = O.time_mix_step(S, r, k, v, w, u)
    assert torch.allclose(o, S.sum(0) + 2 * 0.6 * v)                                            # the old state and the bonus, not the new write
    assert torch.allclose(S2, torch.tensor([[0.5 + 1.8, 1.0 - 1.2], [2.4, -0.25 - 1.6]], dtype=D))
    hist, c = O.conv_step(torch.tensor([[1.0], [2.0]], dtype=D), torch.tensor([3.0], dtype=D), torch.tensor([[10.0, 100.0, 1000.0]], dtype=D), torch.tensor([7.0], dtype=D))
    assert float(c) == 10 + 200 + 3000 + 7 and hist.flatten().tolist() == [2.0, 3.0]
    n = O.part_norm(torch.tensor([3.0, 4.0, 0.0, 2.0], dtype=D), 2, 0.0)
    assert torch.allclose(n, torch.tensor([3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0.0, math.sqrt(2.0)], dtype=D))


def test_routing_by_hand():
    z = torch.tensor([1.0, -9.0, 3.0, 2.0], dtype=D)
    idx, wt = O.route(z, 2)
    e = math.exp(1.0)
    assert idx == [2, 3] and torch.allclose(wt, torch.tensor([e / (1 + e), 1 / (1 + e)], dtype=D))     # softmax over the chosen only
    assert O.route(torch.zeros(4, dtype=D), 2)[0] == [0, 1]


@pytest.mark.parametrize("rank", [1, 8])
def test_whole_model_shapes_loop_and_causality(rank):
    cfg = small_cfg()
    weights = import_module("aws-k8s-ansible-provisioner_b200.weights")
    assert weights.resitar_tensor_shapes(cfg, rank) == O.tensor_shapes(cfg, rank)
    assert {k: tuple(v.shape) for k, v in weights.resitar_random_state_dict(cfg, rank=rank).items()} == O.tensor_shapes(cfg, rank)
    w = O.random_weights(cfg, seed=6, rank=rank)
    toks = [3, 30, 7, 7, 1, 12, 25, 0, 9, 18, 4]
    logits, streams = O.forward(cfg, w, toks)
    assert O.run_order(cfg) == [0, 1, 2, 1, 2, 3]
    assert streams.shape == (6, len(toks), 12) and logits.shape == (len(toks), 31) and torch.isfinite(logits).all()
    assert torch.allclose(O.forward(cfg, w, toks[:6])[0], logits[:6], atol=1e-12)
    assert O.Stepper(cfg, w).greedy(toks[:4], 3)[0] == int(torch.argmax(logits[3]))
    # the streams are not copies of one another: with their mixes exchanged the model is another one
    w2 = dict(w, **{"l1.hc1.mix": w["l1.hc1.mix"].T.contiguous()})
    assert (O.forward(cfg, w2, toks)[0] - logits).abs().max() > 1e-4
