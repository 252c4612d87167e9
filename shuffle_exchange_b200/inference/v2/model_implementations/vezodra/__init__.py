from .policy import VezodraPolicy  # noqa: F401
