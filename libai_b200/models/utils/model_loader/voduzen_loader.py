"""Voduzen checkpoints (``config.json`` + ``model.safetensors``) → :class:`libai_b200.models.VoduzenForCausalLM`.

``config.json``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``logit_scale`` and ``layers`` (per entry ``type``, ``mixer`` sizes and
constants, ``mlp``: ``{kind: moe, expert: {ff}, router: {experts, top, identity}, shared: {ff}}`` or null).  Tensor names: ``embed``,
``final.norm``, ``head`` and per entry ``l<i>.norm1|norm2``, ``l<i>.mix.q`` or ``l<i>.mix.dq|dq.norm|uq``, ``l<i>.mix.dkv|dkv.norm|uk|uv|o|sink``,
``l<i>.mlp.router|correction``, ``l<i>.mlp.e<j>.up|down`` and ``l<i>.mlp.shared.up|down|sg``.  Linear weights are ``[out, in]``; the experts'
matrices are stacked into ``up`` ``[E, ff, width]`` and ``down`` ``[E, width, ff]``.
"""
import collections
import re

import torch

from .base_loader import ModelLoaderHuggerFace

_TOP = {"embed": "model.embed", "final.norm": "model.final_norm.weight", "head": "head"}


class VoduzenLoader(ModelLoaderHuggerFace):
    def _load_config_from_json(self, config_file):
        cfg = self._read_config_json()
        for key in ("vocab", "width", "layers", "norm", "embedding", "logit_scale", "kv_page_size"):
            if key in cfg:
                self._update_cfg(key, cfg[key])
        for key in ("bos_token_id", "eos_token_id", "pad_token_id"):
            if cfg.get(key) is not None:
                self._update_cfg(key, cfg[key])

    def _convert_state_dict(self, sd, cfg):
        out = collections.OrderedDict()
        experts = collections.defaultdict(dict)                # (block, matrix) -> {expert: tensor}
        for name, t in sd.items():
            if name in _TOP:
                out[_TOP[name]] = t
                continue
            m = re.fullmatch(r"l(\d+)\.(.+)", name)
            if not m:
                out[name] = t                                  # reported as unexpected by the base loader
                continue
            i, rest = m.group(1), m.group(2)
            pre = f"model.layers.{i}."
            if rest in ("norm1", "norm2"):
                out[pre + rest + ".weight"] = t
                continue
            m = re.fullmatch(r"mlp\.e(\d+)\.(up|down)", rest)
            if m:
                experts[(i, m.group(2))][int(m.group(1))] = t
                continue
            if rest in ("mlp.router", "mlp.correction"):
                out[pre + rest] = t
                continue
            m = re.fullmatch(r"mlp\.shared\.(up|down|sg)", rest)
            if m:
                out[f"{pre}shared.{m.group(1)}"] = t
                continue
            m = re.fullmatch(r"mix\.(.+)", rest)
            if m:
                out[f"{pre}mix.{m.group(1).replace('.', '_')}"] = t
                continue
            out[name] = t
        for i in sorted({i for i, _ in experts}):
            up, down = experts[(i, "up")], experts[(i, "down")]
            order = sorted(up)
            if order != list(range(len(order))) or sorted(down) != order:
                raise ValueError(f"block {i}: the experts' tensors are not e0 … e{len(order) - 1} with up and down each")
            out[f"model.layers.{i}.mlp.up"] = torch.stack([up[e] for e in order])
            out[f"model.layers.{i}.mlp.down"] = torch.stack([down[e] for e in order])
        return out

    def _load(self, model, state_dict):
        """Every parameter of the model must come from the checkpoint: a tensor that is missing would otherwise stay at its
        random initial value."""
        missing = sorted(set(model.state_dict().keys()) - set(state_dict.keys()))
        if missing:
            raise RuntimeError(f"the checkpoint at {self.pretrained_model_path} lacks tensors for: {missing}")
        return super()._load(model, state_dict)
