"""Opening a model directory for serving: builds what the model's class needs (once), makes the context, loads the model.
One sequence is live at a time; `Session` keeps its id and position and hands its caches and states back."""
from __future__ import annotations

import json
from pathlib import Path

from . import Context, LithosError, LB_ERR_INVALID, LB_ERR_STATE, build
from . import model as M


def open_model(model_dir, max_ctx: int, dtype: str = "bfloat16", device: int = 0):
    """(context, model) of a model directory; the host library and the kernel images the model's class launches are compiled
    in-tree when they are missing or out of date"""
    text = (Path(model_dir) / "config.json").read_text()
    build(images=[])
    images = M.config_images(text)
    if images is None:
        name = json.loads(text).get("architecture")
        raise LithosError(LB_ERR_INVALID, f"no model class for architecture {name!r} (known: {', '.join(M.architectures())})")
    build(images=images)
    ctx = Context(device, images=images)
    try:
        return ctx, M.Model.open(ctx, model_dir, max_ctx, dtype)
    except Exception:
        ctx.close()
        raise


class Session:
    """The one live sequence of a model: portions go in, logits come out; ending it frees the model's caches and states."""

    def __init__(self, model: M.Model):
        self.model, self.id, self.pos = model, None, 0

    def feed(self, seq_id, tokens, want=()):
        """the next tokens of sequence seq_id: logits [len(want), vocab] at these places of the portion"""
        if self.id is None:
            self.model.reset_state()
            self.id, self.pos = seq_id, 0
        elif self.id != seq_id:
            raise LithosError(LB_ERR_STATE, f"sequence {self.id!r} is still live")
        out = self.model.forward(tokens, self.pos, want)
        self.pos += len(tokens)
        return out

    def end(self, seq_id):
        if self.id == seq_id:
            self.id = None
