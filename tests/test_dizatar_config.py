"""Host-side tests of the Dizatar configuration, its model plan, the tensors the plan asks for, its cache
needs and the plain implementation's own mechanisms (no GPU)."""

import copy

import pytest
import torch

import dizatar_tiny as dz
import plain_dizatar as plain
from freetoken_b200.cache import CacheManager, PagedKeyNeed
from freetoken_b200.config.dizatar import DizatarConfig, build_plan
from freetoken_b200.config.model_plan import ConfigError, ModelPlan, RunEntry
from freetoken_b200.csrc import ops
from freetoken_b200.models.model import Model
from freetoken_b200.parts.base import Segment, StepShape
from freetoken_b200.registry import architecture_of
from freetoken_b200.weights.loader import WeightError, plan_loading
from freetoken_b200.weights.spec import leaves


def test_registry_picks_the_design_by_its_singular_key():
    arch = architecture_of(dz.DZ_A)
    assert arch.name == "Dizatar"
    cfg = arch.read_config(dz.DZ_A)
    assert isinstance(cfg, DizatarConfig) and cfg.to_dict() == dz.DZ_A


@pytest.mark.parametrize("which", list(dz.DZ))
def test_plan_hands_every_constant_to_a_part(which):
    raw = dz.DZ[which]
    plan = build_plan(DizatarConfig.from_dict(raw))
    order = plain.run_order(raw)
    assert [(s.layer, s.stream_map == 0) for s in plan.schedule] == order
    assert all(s.owns_cache for s in plan.schedule)
    assert [m.kind for m in plan.stream_maps] == (["embedding_mix"] if raw.get("loop") else [])
    assert plan.head.params["softcap"] == raw.get("logit_softcap", 0.0) and plan.head.params["tied_to"] is None
    for spec, layer in zip(plan.layers, raw["layers"]):
        assert spec.block.kind == "sandwich" and spec.block.params["residual_mult"] == raw.get("residual_mult", 1.0)
        norms = spec.all_norms()
        want = {"mixer": ("norm1", None), "mixer_out": ("norm1b", "ls1")}
        if layer["mlp"]:
            want.update({"feed_forward": ("norm2", None), "feed_forward_out": ("norm2b", "ls2")})
        assert {k: (n.params["tensor"], n.params["scale_tensor"]) for k, n in norms.items()} == want
        assert all(n.params["eps"] == raw["norm"]["eps"] and not n.params["plus_one"] for n in norms.values())
        m, p = layer["mixer"], spec.mixer.params
        assert (p["num_heads"], p["qk_dim"], p["rot_dim"], p["v_dim"], p["rank"], p["sm_scale"], p["output_gate"],
                p["norm_eps"]) == \
            (m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], False, raw["norm"]["eps"])
        if m["rot_dim"]:
            assert (p["position"].kind, p["position"].params["theta"], p["position"].params["rotary_dim"]) == \
                ("rotary_neox", m["rot"]["base"], m["rot_dim"])
        if layer["mlp"]:
            f, r = spec.feed_forward.params, layer["mlp"]["router"]
            assert (f["num_experts"], f["top_k"], f["identity"], f["intermediate_size"]) == \
                (r["experts"], r["top"], r["identity"], layer["mlp"]["expert"]["ff"])
            assert (f["scoring"], f["use_bias"], f["renormalize"], f["scale"]) == ("softmax", True, True, 1.0)
            shared = layer["mlp"].get("shared")
            assert (f["shared"].params["intermediate_size"] if f["shared"] else None) == (shared["ff"] if shared else None)
        else:
            assert spec.feed_forward is None


@pytest.mark.parametrize("which", list(dz.DZ))
def test_the_plan_asks_for_exactly_the_tensors_of_a_checkpoint(which):
    raw = dz.DZ[which]
    model = Model(build_plan(DizatarConfig.from_dict(raw)))
    asked = {}
    for spec in model.tensor_specs():
        for leaf in leaves(spec.all_sources()[0]):
            asked[leaf.name] = tuple(leaf.shape)
    assert asked == plain.expected_tensors(raw)
    shapes = dict(asked)
    plan_loading(model.tensor_specs(), shapes)
    del shapes["l0.ls1"]
    shapes["l0.mix.stranger"] = (3,)
    with pytest.raises(WeightError) as err:
        plan_loading(model.tensor_specs(), shapes)
    assert "l0.ls1" in err.value.missing and "l0.mix.stranger" in err.value.unexpected


def test_every_pass_has_a_cache_of_rows_of_latent_plus_rotated_part():
    raw = dz.DZ_A
    model = Model(build_plan(DizatarConfig.from_dict(raw)))
    needs = model.cache_needs()
    order = [i for i, _ in plain.run_order(raw)]
    assert order == [0, 1, 2, 1, 2, 3] and len(needs) == 6
    for need, i in zip(needs, order):
        m = raw["layers"][i]["mixer"]
        assert need == PagedKeyNeed(1, m["kv_rank"] + m["rot_dim"], None)
    cache = CacheManager(needs, 4, 20, 2, 64)
    cache.admit("a")
    cache.grow("a", 30)
    cache.advance("a", 30)
    cache.release("a")
    assert cache.free_pages() == cache.total_pages()


def _broken(path, value):
    raw = copy.deepcopy(dz.DZ_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return raw


@pytest.mark.parametrize("path,value,match", [
    (("vocab",), KeyError, "vocab"), (("width",), 0, "width"), (("norm", "eps"), KeyError, "eps"),
    (("layers",), [], "layers"), (("layers", 0, "type"), "attention", "type"),
    (("layers", 0, "mixer", "kv_rank"), KeyError, "kv_rank"), (("layers", 1, "mixer", "heads"), 0, "heads"),
    (("layers", 0, "mixer", "rot"), KeyError, "rot"), (("layers", 0, "mixer", "rot", "dims"), 4, "rot.dims"),
    (("layers", 0, "mixer", "rot_dim"), 3, "rot"), (("layers", 0, "mixer", "kv_rank"), 1020, "1024"),
    (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mlp", "router", "top"), 8, "top"),
    (("layers", 0, "mlp", "expert"), KeyError, "expert"), (("layers", 0, "mlp", "router", "identity"), -1, "identity"),
    (("layers", 0, "mlp", "shared", "ff"), 0, "shared"), (("loop", "stop"), 1, "loop"), (("loop", "stop"), 9, "loop"),
    (("loop", "times"), 0, "loop"), (("loop", "start"), KeyError, "start"), (("logit_softcap",), -1.0, "softcap")])
def test_a_bad_config_names_the_key(path, value, match):
    with pytest.raises(ConfigError, match=match):
        DizatarConfig.from_dict(_broken(path, value))


def test_a_stream_map_must_exist_and_wants_the_plain_residual():
    plan = build_plan(DizatarConfig.from_dict(dz.DZ_A))
    parts = {f: getattr(plan, f) for f in plan.__dataclass_fields__}
    with pytest.raises(ValueError, match="stream map"):
        ModelPlan(**{**parts, "schedule": (RunEntry(0, stream_map=1),)}).validate()
    with pytest.raises(ValueError, match="stream"):
        ModelPlan(**{**parts, "residual_streams": 2}).validate()


def test_step_plan_of_the_two_forms():
    """Portions of 64 tokens and more take the expanded form, the rest row tiles of the absorbed one; every
    query token and every context row is listed once."""
    model = Model(build_plan(DizatarConfig.from_dict(dz.DZ_B)))
    mixer = model.blocks[0].mixer
    assert mixer.step_plan_key() == "paged_attention"             # before the weights are bound: not decided
    assert mixer._takes_own_kernels(torch.bfloat16) and mixer._expands(torch.bfloat16)
    assert not mixer._takes_own_kernels(torch.float32)
    mixer.own_kernels = mixer.expands = True
    segs = [Segment(0, 9, 1, 0), Segment(1, 130, 70, 1), Segment(2, 0, 63, 71), Segment(3, 0, 300, 134)]
    plan = mixer.plan_step(StepShape(segs, 434, 64, 8, 300, 300))
    a, H = plan.arrays, mixer.nq
    rt = ops.latent_row_tile(H, mixer.d, mixer.rank)
    assert list(zip(a["flat_seg"], a["flat_row"])) == [(0, 0)] + [(2, r) for r in range(0, 63 * H, rt)]
    assert plan.host["flat_tokens"] == (0, 134) and plan.host["flat_kv"] == 63
    assert list(zip(a["x_seg"], a["x_q0"], a["x_row0"])) == [(1, 0, 0), (3, 0, 256), (3, 128, 256), (3, 256, 256)]
    assert plan.host["rows"] == 256 + 320 and len(a["g_seg"]) == 9
    assert [int(r) for r in a["g_row0"]] == list(range(0, 576, 64))
    decode = mixer.plan_step(StepShape([Segment(0, 99, 1, 0)], 1, 64, 8, 1, 100))
    assert decode.host["flat_kv"] == 512 and decode.host["expanded"] == 0


def test_splits_cover_the_keys():
    for tiles in (1, 8, 64, 500):
        for kv in (1, 64, 65, 2048, 30000):
            n, per = ops.latent_splits(tiles, kv, 148)
            assert per % 64 == 0 and (n - 1) * per < kv <= n * per and n <= 64


# ------------------------------------------------------------- the plain implementation itself
def test_plain_identity_experts_and_correction():
    config = dz.one_layer(dz.layer(2, 4, 2, 4, 6, dz.moe(3, 2, 8, identity=2, shared=8)), width=12)
    w = dz.random_state(config, 5)
    h = torch.randn(7, 12, dtype=torch.float64)
    mlp = config["layers"][0]["mlp"]
    w["l0.mlp.correction"] = torch.tensor([0.0, 0.0, 0.0, 50.0, 40.0], dtype=torch.float64)
    ids, s = plain.choose_experts(h, w, "l0.mlp.", mlp["router"])
    assert bool((ids == torch.tensor([3, 4])).all())
    # both chosen hand the input back and the weights add up to one, whatever the correction
    out = plain.routed_ff(h, w, "l0.mlp.", mlp) - plain.glu(h, w, "l0.mlp.shared.")
    assert torch.allclose(out, h)
    assert torch.allclose(s.sum(-1), torch.ones(7, dtype=torch.float64))


def test_plain_loop_maps_the_stream_before_every_pass():
    config = dz.model(30, 12, [dz.layer(2, 4, 2, 4, 6)], loop=(0, 1, 2))
    w = dz.random_state(config, 6)
    w["l0.ls1"].zero_()                                     # the layer adds nothing: only the maps are left
    x0 = w["embed"][[3, 4]]
    x = x0
    for _ in range(2):
        x = torch.cat([x, x0], -1) @ w["loop.in"].T
    want = plain.rms(x, 1e-6) * w["final.norm"] @ w["head"].T
    assert torch.allclose(plain.forward(config, w, [3, 4]), want)
