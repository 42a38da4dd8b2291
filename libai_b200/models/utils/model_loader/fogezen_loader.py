"""Fogezen checkpoints (``config.json`` + ``model.safetensors``) → :class:`libai_b200.models.FogezenForCausalLM`.

``config.json``: ``vocab``, ``width``, ``norm.eps``, ``residual_mult``, ``embedding.scale``, ``layers`` (per entry ``type``, ``mixer`` sizes and
constants, ``mlp``: ``{kind: dense, ff}`` or null) and ``loop``: ``{start, stop, times}`` or absent.  Tensor names: ``embed``, ``final.norm``,
``loop.step`` and per entry ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mlp.gate|up|down``; mixer ``attention``: ``l<i>.mix.q|k|v`` with ``.b``,
``l<i>.mix.o``; mixer ``parallel``: ``l<i>.mix.left.q|k|v|g|o|q.norm|k.norm|out`` and ``l<i>.mix.right.q|k|v|g|o|i|f|i.b|f.b|norm|out``.  Linear weights
are ``[out, in]``; the feed-forward's ``gate`` and ``up`` are stacked into one ``[2·ff, width]`` matrix.
"""
import collections
import re

import torch

from .base_loader import ModelLoaderHuggerFace

_TOP = {"embed": "model.embed", "final.norm": "model.final_norm.weight", "loop.step": "model.loop_step"}


class FogezenLoader(ModelLoaderHuggerFace):
    def _load_config_from_json(self, config_file):
        cfg = self._read_config_json()
        for key in ("vocab", "width", "layers", "norm", "embedding", "residual_mult", "loop", "kv_page_size"):
            if key in cfg:
                self._update_cfg(key, cfg[key])
        for key in ("bos_token_id", "eos_token_id", "pad_token_id"):
            if cfg.get(key) is not None:
                self._update_cfg(key, cfg[key])

    def _convert_state_dict(self, sd, cfg):
        out = collections.OrderedDict()
        pairs = collections.defaultdict(dict)                  # block -> {"gate" / "up": tensor}
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
            if rest in ("norm1", "norm1b", "norm2", "norm2b"):
                out[pre + rest + ".weight"] = t
            elif rest in ("mlp.gate", "mlp.up"):
                pairs[i][rest[4:]] = t
            elif rest == "mlp.down":
                out[pre + rest] = t
            elif rest in ("mix.left.out", "mix.right.out"):
                out[f"{pre}{rest.replace('.out', '_out')}.weight"] = t
            elif re.fullmatch(r"mix\.(left|right)\..+", rest):
                side, part = rest.split(".", 2)[1:]
                out[f"{pre}mix.{side}.{part.replace('.', '_')}"] = t
            elif rest.startswith("mix."):
                out[f"{pre}mix.{rest[4:].replace('.', '_')}"] = t
            else:
                out[name] = t
        for i, p in pairs.items():
            if set(p) != {"gate", "up"}:
                raise ValueError(f"block {i}: the feed-forward needs both gate and up, the checkpoint has {sorted(p)}")
            out[f"model.layers.{i}.mlp.gate_up"] = torch.cat([p["gate"], p["up"]], 0)
        return out

    def _load(self, model, state_dict):
        """Every parameter of the model must come from the checkpoint: a tensor that is missing would otherwise stay at its
        random initial value."""
        missing = sorted(set(model.state_dict().keys()) - set(state_dict.keys()))
        if missing:
            raise RuntimeError(f"the checkpoint at {self.pretrained_model_path} lacks tensors for: {missing}")
        return super()._load(model, state_dict)
