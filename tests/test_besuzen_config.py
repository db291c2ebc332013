"""Host-side tests of the Besuzen configuration, its model plan, the tensors the plan asks for, the size that
only a checkpoint's tensor shapes state, and the plain implementation's own mechanisms (no GPU)."""

import copy
import json
import os

import pytest
import torch

import besuzen_tiny as bz
import plain_besuzen as plain
from freetoken_b200.cache.manager import CacheManager, CompositeNeed, PagedKVNeed, StateNeed
from freetoken_b200.config.besuzen import BesuzenConfig, build_plan, sizes_from_tensors
from freetoken_b200.config.model_plan import ConfigError
from freetoken_b200.models.model import Model
from freetoken_b200.registry import architecture_of, read_model_config
from freetoken_b200.weights.loader import WeightError, load_tensors, plan_loading


def test_registry_picks_the_design():
    arch = architecture_of(bz.BZ_A)
    assert arch.name == "Besuzen"
    cfg = arch.read_config(bz.BZ_A)
    assert isinstance(cfg, BesuzenConfig) and cfg.to_dict() == bz.BZ_A


@pytest.mark.parametrize("which", list(bz.BZ))
def test_plan_hands_every_constant_to_a_part(which):
    raw = bz.BZ[which]
    plan = build_plan(BesuzenConfig.from_dict(raw))
    assert plan.embedding.params["scale"] == raw["embedding"]["scale"]
    assert plan.final_norm.params["factor"] == raw["logit_scale"]
    assert [s.layer for s in plan.schedule] == list(range(len(raw["layers"])))
    mixing = [i for i, l in enumerate(raw["layers"]) if l["type"] == "attention" and l["mixer"]["v_mix"]]
    for i, (spec, layer) in enumerate(zip(plan.layers, raw["layers"])):
        m, mlp = layer["mixer"], layer["mlp"]
        assert sorted(spec.all_norms()) == (["feed_forward", "mixer"] if mlp else ["mixer"])
        assert all(n.params["eps"] == raw["norm"]["eps"] for n in spec.all_norms().values())
        if layer["type"] == "attention":
            left, p = m, spec.mixer.params
            assert p["gate"] == "element" and p["position"].get("rotary_dim", 0) == m["rot"]["dims"]
            if m["rot"]["dims"]:
                assert p["position"].kind == "rotary_interleaved" and p["position"].params["theta"] == m["rot"]["base"]
            assert p["value_mix"] == (None if i not in mixing else "source" if i == mixing[0] else "blend")
        else:
            left, right = m["left"], m["right"]
            p, r = (part.params for part in spec.mixer.params["members"])
            assert spec.mixer.params["scales"] == (m["left_scale"], m["right_scale"])
            assert p["gate"] == "head" and p["value_mix"] is None and p["position"].kind == "none"
            assert (r["heads"], r["key_dim"], r["head_dim"], r["low_rank"]) == (right["heads"], right["dim"], right["dim"],
                                                                                right["low_rank"])
            assert r["norm_eps"] == raw["norm"]["eps"]
        assert (p["num_heads"], p["num_kv_heads"], p["head_dim"], p["value_dim"], p["sm_scale"]) == (
            left["heads"], left["kv_heads"], left["dim"], left["vdim"], left["scale"])
        assert p["bias"] and not p["o_bias"]
        if mlp and mlp["kind"] == "dense":
            f = spec.feed_forward.params
            assert (f["intermediate_size"], f["activation"], f["gated"]) == (mlp["ff"], "gelu_tanh", True)
        elif mlp:
            f, r = spec.feed_forward.params, mlp["router"]
            assert (f["num_experts"], f["top_k"], f["groups"], f["keep_groups"], f["group_top"]) == (
                r["experts"], r["top"], r["groups"]["count"], r["groups"]["keep"], 1)
            assert (f["scoring"], f["use_bias"], f["renormalize"], f["scale"]) == ("softmax", False, True, 1.0)
            assert f["intermediate_size"] == mlp["expert"]["ff"] and f["activation"] == "silu"
            if mlp.get("shared"):
                s = f["shared"].params
                assert f["shared_gate"] and (s["intermediate_size"], s["activation"]) == (mlp["shared"]["ff"], "silu")
            else:
                assert f["shared"] is None and not f["shared_gate"]


@pytest.mark.parametrize("which", list(bz.BZ))
def test_the_plan_asks_for_exactly_the_tensors_of_a_checkpoint(which):
    raw = bz.BZ[which]
    shapes = plain.expected_tensors(raw)
    specs = Model(build_plan(BesuzenConfig.from_dict(raw))).tensor_specs()
    plan_loading(specs, shapes)                                    # complete, nothing unexpected, every shape right
    for name in shapes:
        rest = {k: v for k, v in shapes.items() if k != name}
        first = min((int(k[1:].split(".")[0]) for k in shapes if k.endswith("vmix")), default=-1)
        if name == f"l{first}.mix.vmix":
            plan_loading(specs, rest)                              # the first mixing layer's factor is unused
            continue
        with pytest.raises(WeightError) as err:
            plan_loading(specs, rest)
        assert err.value.missing == [name]
    with pytest.raises(WeightError) as err:
        plan_loading(specs, {**shapes, "l0.mix.extra": (3,)})
    assert err.value.unexpected == ["l0.mix.extra"]


def test_a_folder_states_the_middle_of_the_decay_projection(tmp_path):
    """config.json without it: the checkpoint's shapes fill it in; the loaded tensors are the folder's."""
    folder = bz.write_tiny(str(tmp_path / "m"), "A")
    with open(os.path.join(folder, "config.json")) as f:
        assert "low_rank" not in f.read()
    arch, cfg = read_model_config(folder)
    assert [l.mixer.right.low_rank for l in cfg.layers if l.type == "parallel"] == [5, 1]
    model = Model(arch.build_plan(cfg))
    tensors = load_tensors(model.tensor_specs(), folder, torch.float32, "cpu", arch.rename_tensor)
    state = bz.random_state(bz.BZ_A, bz.SEEDS["A"])
    assert torch.equal(tensors["l0.mix.right.rkvg"].double(), torch.stack([state[f"l0.mix.right.{n}"] for n in "rkvg"]))
    assert torch.equal(tensors["l0.mlp.router_sg"].double(), torch.cat([state["l0.mlp.router"], state["l0.mlp.shared.sg"]]))
    assert tensors["l3.mix.vmix"].shape == () and "l1.mix.vmix" not in tensors
    model.bind(tensors, torch.float32)
    assert torch.allclose(model.final_norm.weight.double(), state["final.norm"] * bz.BZ_A["logit_scale"])
    # the gate's rows of the merged product are added no bias
    mixer = model.blocks[1].mixer
    assert mixer.b_qkv.numel() == mixer.w_qkv.shape[0] and float(mixer.b_qkv[-mixer.nq * mixer.d:].abs().max()) == 0
    with pytest.raises(ConfigError, match="low_rank"):
        BesuzenConfig.from_dict(json.loads(json.dumps(bz.file_config(bz.BZ_A))))
    filled = sizes_from_tensors(bz.file_config(bz.BZ_A), plain.expected_tensors(bz.BZ_A))
    assert BesuzenConfig.from_dict(filled).layers == BesuzenConfig.from_dict(bz.BZ_A).layers


@pytest.mark.parametrize("dtype,d", [(torch.float32, 48), (torch.bfloat16, 64)])
def test_cache_needs(dtype, d):
    """Attention keeps keys and values in pages (heads filled up for the tensor-core kernels in bfloat16), a
    parallel mixer beside them the previous input and the state in a slot."""
    raw = bz.several([bz.attention(4, 2, 40, 48, 8), bz.parallel((2, 1, 40, 48), (3, 10, 4))], width=48)
    model = Model(build_plan(BesuzenConfig.from_dict(raw)))
    for block in model.blocks:
        for part in (block.mixer, *getattr(block.mixer, "members", [])):
            if hasattr(part, "_head_size"):
                part.d = part._head_size(dtype)
    needs = model.cache_needs()
    assert needs[0] == PagedKVNeed(2, d, None)
    assert needs[1] == CompositeNeed((PagedKVNeed(1, d, None), StateNeed((48 + 3 * 10 * 10,), "float32")))
    manager = CacheManager(needs, page_size=8, num_pages=6, max_slots=2, max_seq_len=48)
    assert len(manager.paged_groups) == 2 and len(manager.state_groups) == 1


BAD = {
    "no scale": (lambda c: c["layers"][1]["mixer"].pop("scale"), "layers\\[1\\].mixer.scale"),
    "no rotation": (lambda c: c["layers"][1]["mixer"].pop("rot"), "layers\\[1\\].mixer.rot"),
    "odd rotation": (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "rot.dims"),
    "rotation wider than a head": (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "rot.dims"),
    "key heads": (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    "unknown mixer": (lambda c: c["layers"][0].update(type="conv"), "type"),
    "unknown feed-forward": (lambda c: c["layers"][1]["mlp"].update(kind="relu"), "mlp.kind"),
    "no left": (lambda c: c["layers"][0]["mixer"].pop("left"), "mixer.left"),
    "no right": (lambda c: c["layers"][0]["mixer"].pop("right"), "mixer.right"),
    "groups do not divide": (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    "groups too small": (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "top"),
    "more than there are": (lambda c: c["layers"][3]["mlp"]["router"].update(top=5), "top"),
    "values that do not fit": (lambda c: c["layers"][3]["mixer"].update(vdim=12), "blends its values"),
    "no layers": (lambda c: c.update(layers=[]), "layers"),
    "eps": (lambda c: c["norm"].update(eps=-1.0), "norm.eps"),
}


@pytest.mark.parametrize("what", list(BAD))
def test_a_bad_configuration_names_the_key(what):
    change, key = BAD[what]
    raw = copy.deepcopy(bz.BZ_A)
    change(raw)
    with pytest.raises(ConfigError, match=key):
        BesuzenConfig.from_dict(raw)


def test_defaults():
    """Absent scales are 1, an absent value size is the key size, absent groups are one group of all."""
    raw = copy.deepcopy(bz.BZ_A)
    raw.pop("embedding"), raw.pop("logit_scale")
    raw["layers"][1]["mixer"].pop("vdim"), raw["layers"][3]["mixer"].update(vdim=12)
    raw["layers"][3]["mlp"]["router"].pop("groups")
    cfg = BesuzenConfig.from_dict(raw)
    assert (cfg.embedding_scale, cfg.logit_scale) == (1.0, 1.0)
    assert cfg.layers[1].mixer.vdim == 12
    assert (cfg.layers[3].mlp.groups, cfg.layers[3].mlp.keep) == (1, 1)


# ------------------------------------------------------------- the plain implementation itself
def test_plain_is_causal_and_scales_its_logits():
    state = bz.random_state(bz.BZ_A, 3)
    toks = bz.tokens(4, 20, 150)
    full = plain.forward(bz.BZ_A, state, toks)
    assert torch.allclose(plain.forward(bz.BZ_A, state, toks[:11]), full[:11], atol=1e-10)
    twice = {**bz.BZ_A, "logit_scale": 2 * bz.BZ_A["logit_scale"]}
    assert torch.allclose(plain.forward(twice, state, toks), 2 * full)


def test_plain_group_choice():
    """The best expert sits in a group that is dropped when another group's best is larger."""
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    z = torch.tensor([1.0, 0.9, 3.0, -5.0, 2.9, 2.8], dtype=torch.float64)
    ids, w, margin = plain.choose_experts(z, router)
    s = torch.softmax(z, -1)
    assert ids == [2, 3] and torch.allclose(w, s[[2, 3]] / s[[2, 3]].sum())
    assert margin == pytest.approx(float(s[2] - s[4]))
    ids, _, _ = plain.choose_experts(z, {**router, "groups": {"count": 3, "keep": 2}})
    assert ids == [2, 4]


def test_plain_time_mixing_by_hand():
    """Two tokens, one head of one channel: the bonus counts for the current token only."""
    one = torch.ones(2, 1, 1, dtype=torch.float64)
    r, k, v, w = 2 * one, one * torch.tensor([3.0, 5.0], dtype=torch.float64).view(2, 1, 1), 7 * one, 0.5 * one
    o = plain.time_mixing_scan(r, k, v, w, torch.full((1, 1), 0.1, dtype=torch.float64))
    assert o[0, 0, 0] == pytest.approx(2 * 0.1 * 3 * 7) and o[1, 0, 0] == pytest.approx(2 * (21 + 0.1 * 5 * 7))
